"""Zevedra's configuration and its place in the registries, and the plain implementation's pieces against direct
arithmetic (no GPU)."""
import copy
import math

import numpy as np
import pytest
import torch

import helpers
import plain_zevedra as plain
import zevedra_helpers as zh
from sprout_lm_b200.config import ConfigError, ZevedraConfig, parse_config, registered_architectures
from sprout_lm_b200.config.specs import PartSpec
from sprout_lm_b200.models.decoder import DecoderModel
from sprout_lm_b200.parts import StateView, build_part
from sprout_lm_b200.weights.random_init import random_tensor


def test_registered_and_round_trip():
    assert "Zevedra" in registered_architectures()
    for raw, _, _ in zh.CONFIGS.values():
        config = parse_config(raw)
        assert isinstance(config, ZevedraConfig)
        assert parse_config(config.to_dict()) == config
        assert config.to_dict() == raw


def test_model_spec_follows_the_file():
    spec = parse_config(zh.A).model_spec()
    assert [layer.block for layer in spec.layers] == ["pre_norm"] * 4
    assert all(layer.mixer.kind == "parallel_mixers" and layer.options["branch_scale"] == 0.9 for layer in spec.layers)
    assert [layer.feed_forward.kind for layer in spec.layers] == ["routed_experts", "none", "routed_experts", "routed_experts"]
    assert [len(layer.norms) for layer in spec.layers] == [2, 1, 2, 2]
    windowed, delta = spec.layers[0].mixer.params["mixers"]
    assert spec.layers[0].mixer.params["scales"] == (0.7, 1.1) and "norms" not in spec.layers[0].mixer.params
    assert windowed.params["mask"] == ("window", 5) and windowed.params["conv"] == 3 and windowed.params["gate"] == "head"
    assert windowed.params["position"].kind == windowed.params["value_position"].kind == "rope_interleaved"
    assert windowed.params["position"].params["dims"] == 4 and windowed.params["value_position"].params["dims"] == 10
    assert delta.kind == "gated_delta_rule" and delta.params["kv_heads"] == 1 and delta.params["taps"] == 2
    full, writer = spec.layers[1].mixer.params["mixers"]
    assert spec.layers[1].mixer.params["norms"] == ("mix.left.out", "mix.right.out") and spec.layers[1].mixer.params["scales"] == (0.5, 0.5)
    assert full.params["unit_sink"] and full.params["qk_norm_span"] == "projection" and full.params["gate"] == "element"
    assert full.params["position"].kind == "rope_yarn" and "mask" not in full.params and full.params["scale"] == 0.6
    assert writer.kind == "forget_write_attention"
    routed = spec.layers[0].feed_forward.params
    assert routed["scores"] == "sigmoid" and routed["weight_on"] == "input" and routed["expert_kind"] == "silu_glu" and routed["top"] == 2
    # layers 1 and 2 run three times: every run has a cache slot and a state entry of its own
    assert [(c.layer, c.cache) for c in spec.order] == [(0, 0), (1, 1), (2, 2), (1, 4), (2, 5), (1, 6), (2, 7), (3, 3)]
    assert spec.stream.kind == "loop_restart" and spec.stream.params["starts"] == (1, 3, 5)
    model = DecoderModel(spec)
    caches = model.cache_specs()
    assert (caches[0].kind, caches[0].window, caches[0].head_dim, caches[0].value_dim) == ("window", 5, 6, 10)
    assert all(caches[i].kind == "full" and caches[i].kv_heads == 3 for i in (1, 4, 6)) and caches[5].window == 9
    states = model.state_specs()
    assert [s.shape for s in states[0]] == [(2, 4 * 6 + 2 * 6 + 2 * 10), (1, 2 * 7 + 3 * 5), (3, 7, 5)]
    assert states[1].shape == (2, 5, 9) and states[4].shape == (2, 5, 9) and states[3].shape == (3, 12, 4)
    assert [s.shape for s in states[7]] == [(1, 40), (3, 2 * 2 * 4 + 22), (2, 4, 11)]
    assert len(states) == 9 and states[8].shape == (1,) and states[8].dtype == torch.int32          # the embedding's last token
    names = {decl.name: decl.shape for decl in model.tensor_decls()}
    assert names["embed"] == (203, 36) and names["bigram"] == (98, 36) and names["head"] == (203, 36) and names["loop.step"] == (3, 36)
    assert names["l0.norm1"] == names["l0.norm2"] == names["final.norm"] == () and "l1.norm2" not in names
    assert names["l0.mix.left.q.conv"] == (24, 3) and names["l0.mix.left.g"] == (4, 36) and names["l0.mix.left.o"] == (36, 40)
    assert names["l0.mix.right.q"] == (7, 36) and names["l0.mix.right.v.conv"] == (15, 2) and names["l0.mix.right.A_log"] == (3,)
    assert names["l0.mix.right.dt_bias"] == (3,) and names["l0.mix.right.norm"] == (5,) and names["l0.mix.right.g"] == (15, 36)
    assert names["l1.mix.left.q.norm"] == (24,) and names["l1.mix.left.k.norm"] == (24,) and names["l1.mix.left.g"] == (18, 36)
    assert names["l1.mix.right.lower"] == names["l1.mix.right.f.b"] == (10,) and names["l1.mix.left.out"] == (36,)
    assert names["l0.mlp.router"] == (5, 36) and names["l0.mlp.e4.gate"] == (12, 36) and names["l0.mlp.e4.down"] == (36, 12)
    assert "l1.mlp.router" not in names and "l0.mix.left.q.norm" not in names and "l1.mix.left.q.conv" not in names


def test_a_model_without_loop_or_pairs():
    spec = parse_config(zh.B).model_spec()
    assert spec.stream is None and spec.embedding.kind == "token_embedding" and spec.embedding.params["scale"] == 0.5
    model = DecoderModel(spec)
    assert model.state_specs()[-1] is None
    assert spec.layers[1].mixer.params["mixers"][0].params["position"].kind == "none"
    names = {decl.name: decl.shape for decl in model.tensor_decls()}
    assert "bigram" not in names and "loop.step" not in names
    assert names["l1.mix.right.q.conv"] == (32, 1) and names["l2.mix.left.k.conv"] == (16, 1)
    # a single tap keeps one (unused) input: the kernel's least
    assert [s.shape for s in model.state_specs()[1]] == [(5, 64 + 64 + 64), (1, 32 + 32 + 96), (4, 16, 24)]


def test_factors_reach_the_parts():
    """The layer's multiplier and the mixers' scales are folded into the parts; a normed pair keeps them for its own kernel."""
    model = DecoderModel(parse_config(zh.A).model_spec())
    pair = model.blocks[0].mixer
    assert pair.mixers[0].out_scale == pytest.approx(0.7 * 0.9) and pair.mixers[1].out_scale == pytest.approx(1.1 * 0.9)
    normed = model.blocks[1].mixer
    assert [m.out_scale for m in normed.mixers] == [1.0, 1.0] and normed.scales == pytest.approx((0.45, 0.45))
    assert model.blocks[0].feed_forward.out_scale == pytest.approx(0.9) and model.blocks[1].feed_forward is None


def test_states_of_two_mixers_side_by_side():
    """Each mixer of a pair gets the views of its own state tensors."""
    pair = DecoderModel(parse_config(zh.A).model_spec()).blocks[0].mixer
    buffers = tuple(torch.zeros(4, *s.shape) for s in pair.state_spec())
    state = StateView(buffers, torch.tensor([2]))
    assert pair._state_of(0, state).buffer is buffers[0]
    own = pair._state_of(1, state)
    assert own.part(0).buffer is buffers[1] and own.part(1).buffer is buffers[2] and own.slots is state.slots
    single = DecoderModel(parse_config(zh.A).model_spec()).blocks[1].mixer
    alone = StateView(torch.zeros(4, 2, 5, 9), torch.tensor([1]))
    assert single._state_of(0, alone) is None and single._state_of(1, alone) is alone


def test_random_values_of_new_kinds():
    assert random_tensor(1, "n", (), "gain").shape == () and 0.8 < float(random_tensor(1, "n", (), "gain")) < 1.2
    share = random_tensor(2, "s", (500,), "share")
    assert float(share.min()) >= 0.0 and float(share.max()) <= 0.95 and 0.1 < float(share.std()) < 0.3


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0]["mixer"]["left"].__setitem__("heads", 5), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["right"].__setitem__("kv_heads", 2), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].__setitem__("dims", 8), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"].__setitem__("vdim", 9), "vdim must be even"),
    (lambda c: c["layers"][0]["mixer"]["left"].__setitem__("conv", 9), "at most 8 taps"),
    (lambda c: c["layers"][0]["mixer"]["right"].__setitem__("conv", 0), "conv"),
    (lambda c: c["layers"][0]["mixer"]["right"].__setitem__("dim", 300), "at most 256"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("mask"), "mask"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1].__setitem__("type", "parallel_3"), "type"),
    (lambda c: c["layers"][3]["mlp"].__setitem__("kind", "dense"), "kind"),
    (lambda c: c["layers"][3]["mlp"]["router"].__setitem__("top", 8), "top"),
    (lambda c: c["embedding"]["bigram"].__setitem__("buckets", 0), "buckets"),
    (lambda c: c["embedding"]["bigram"].__setitem__("mul_cur", 1 << 40), "31 bits"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c["loop"].__setitem__("stop", 5), "loop"),
    (lambda c: c["loop"].__setitem__("times", 0), "loop"),
    (lambda c: c["norm"].__setitem__("eps", 0), "eps"),
    (lambda c: c.__setitem__("vocab", 0), "vocab"),
])
def test_refusals(edit, text):
    raw = copy.deepcopy(zh.A)
    edit(raw)
    with pytest.raises(ConfigError, match=text):
        parse_config(raw)


def test_parts_refuse_what_they_cannot_compute():
    base = {"hidden_size": 16, "heads": 2, "kv_heads": 1, "dim": 4, "value_dim": 4, "scale": 1.0, "position": PartSpec("none", {}), "maps": 1}
    for wrong in ({"gate": "row"}, {"qk_norm_span": "model"}, {"sink": True, "unit_sink": True}, {"conv": 2, "bias": True}, {"conv": 0},
                  {"maps": 2, "conv": 2}, {"own_kv": False, "gate": "element"}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("multimap_attention", {**base, **wrong}))
    moe = {"hidden_size": 16, "experts": 4, "identity": 0, "top": 2, "scale": 1.0, "expert_ff": 8, "expert_kind": "silu_glu", "correction": False}
    build_part("feed_forward", PartSpec("routed_experts", {**moe, "scores": "sigmoid", "weight_on": "input"}))
    for wrong in ({"scores": "relu"}, {"weight_on": "both"}, {"identity": 1, "weight_on": "input"}, {"shared_ff": 4}, {"expert_kind": "swish"}):
        with pytest.raises(ValueError):
            build_part("feed_forward", PartSpec("routed_experts", {**moe, **wrong}))
    two = PartSpec("forget_write_attention", {"hidden_size": 16, "heads": 1, "dim": 4, "value_dim": 4, "eps": 1e-5})
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("parallel_mixers", {"mixers": (two, two), "scales": (0.5, 0.4), "names": ("a.", "b."),
                                                         "norms": ("a.out", "b.out"), "norm_eps": 1e-5, "hidden_size": 16}))


def test_a_lost_state_a_dropped_sink_or_a_shifted_window_shows(tmp_path):
    """The test models are made so that each mechanism matters: a mistake planted in the plain implementation moves the logits
    by far more than the bar."""
    directory = zh.make_model_dir(tmp_path, "A")
    tokens = helpers.random_tokens(np.random.default_rng(31), 60, zh.A["vocab"])
    full = zh.plain_logits(directory, tokens)
    bar = 0.1                              # what 16 bits are allowed, and half as much again

    def moved(other, places=slice(None)):
        """The largest change at any place: a fault is found if one place is over the bar."""
        return max(zh.relative(a, b) for a, b in zip(other, full[places]))
    assert moved(zh.plain_logits(directory, tokens[30:]), slice(30, None)) > bar
    config, tensors = zh.plain_model(directory)

    def with_tensors(change):
        return plain.forward(config, {k: change(k, v) for k, v in tensors.items()}, tokens)
    for label, change in {
            "passes": lambda k, v: np.zeros_like(v) if k == "loop.step" else v,
            "pairs": lambda k, v: np.zeros_like(v) if k == "bigram" else v,
            "first pair": lambda k, v: np.concatenate([v[:-1], v[:1]]) if k == "bigram" else v,
            "decays": lambda k, v: v + 1.0 if k.endswith(".A_log") else v,
            "decay bias": lambda k, v: np.zeros_like(v) if k.endswith(".dt_bias") else v,
            "write strength": lambda k, v: np.zeros_like(v) if k.endswith(".right.b") else v,
            "floors": lambda k, v: np.zeros_like(v) if k.endswith(".lower") else v,
            "forget bias": lambda k, v: np.zeros_like(v) if k.endswith(".f.b") else v,
            "whole norms": lambda k, v: np.ones_like(v) if k.endswith((".q.norm", ".k.norm")) else v,
            "output norms": lambda k, v: np.ones_like(v) if k.endswith(".out") else v,
            "head norms": lambda k, v: np.ones_like(v) if k.endswith(".right.norm") else v,
            "taps": lambda k, v: np.eye(v.shape[1])[-1] * np.ones_like(v) if k.endswith(".conv") else v,
            "gates": lambda k, v: np.zeros_like(v) if k.endswith(".g") else v}.items():
        assert moved(with_tensors(change)) > bar, label
    edits = [lambda c: c["layers"][0]["mixer"]["left"]["mask"].__setitem__("size", 6),
             lambda c: c["layers"][2]["mixer"]["left"]["mask"].__setitem__("size", 8),
             lambda c: c["layers"][0]["mixer"]["left"]["rot"].__setitem__("dims", 6),
             lambda c: c["layers"][2]["mixer"].__setitem__("right_scale", 0.6),
             lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 1),
             lambda c: c["layers"][0].__setitem__("mlp", None),
             lambda c: c.__setitem__("residual_mult", 1.0),
             lambda c: c["embedding"].__setitem__("scale", 1.0),
             lambda c: c["embedding"]["bigram"].__setitem__("mul_prev", 0),
             lambda c: c["loop"].__setitem__("times", 2),
             lambda c: c.__setitem__("loop", None)]
    for number, edit in enumerate(edits):
        changed = copy.deepcopy(config)
        edit(changed)
        assert moved(plain.forward(changed, tensors, tokens)) > bar, number
    # pieces of the mechanisms left out
    real = {key: getattr(plain, key) for key in ("rotate", "softmax_attention", "delta_rule", "forget_and_write", "route", "run_order")}

    def planted(key, fn):
        try:
            setattr(plain, key, fn)
            return moved(plain.forward(config, tensors, tokens))
        finally:
            setattr(plain, key, real[key])
    assert planted("rotate", lambda x, p, b, d, i: x if (np.asarray(p) < 0).any() else real["rotate"](x, p, b, d, i)) > bar      # no turn back
    assert planted("softmax_attention", lambda *a, window=None, unit_sink=False: real["softmax_attention"](*a, window=window)) > bar
    assert planted("delta_rule", lambda q, k, v, g, beta: real["delta_rule"](q, 0 * k + k, v, np.ones_like(g), beta)) > bar
    assert planted("forget_and_write", lambda q, f, v: real["forget_and_write"](q, np.minimum(f, 0.9), v)) > bar
    assert planted("route", lambda h, r, top: (real["route"](h, r, top)[0], np.ones((len(h), top)))) > bar
    assert planted("run_order", lambda c: [(i, t, begins and t == 0) for i, t, begins in real["run_order"](c)]) > bar


# ------------------------------------------------------------------------------------------------ the plain pieces
def test_plain_pieces_against_direct_arithmetic():
    assert plain.softplus(np.array([0.0, 40.0])) == pytest.approx([math.log(2), 40.0])
    # three taps, zeros before the start
    u = np.array([[1.0], [2.0], [4.0], [8.0]])
    assert plain.short_conv(u, np.array([[100.0, 10.0, 1.0]]))[:, 0] == pytest.approx([1.0, 12.0, 124.0, 248.0])
    # a quarter turn at position 1 in both layouts, and what lies beyond the rotated width stays
    x = np.array([[[1.0, 2.0, 3.0, 4.0, 5.0]]])
    turned = plain.rotate(x, np.array([np.pi / 2]), 1e12, 4, True)[0, 0]
    assert turned == pytest.approx([-2.0, 1.0, 3.0, 4.0, 5.0], abs=1e-4)
    assert plain.rotate(x, np.array([np.pi / 2]), 1e12, 4, False)[0, 0] == pytest.approx([-3.0, 2.0, 1.0, 4.0, 5.0], abs=1e-4)
    # turning a value by its place and back by the reader's leaves a turn by the distance
    there = plain.rotate(plain.rotate(x[..., :4], np.array([7]), 30.0, 4, True), np.array([-9]), 30.0, 4, True)
    assert there == pytest.approx(plain.rotate(x[..., :4], np.array([-2]), 30.0, 4, True))
    # a window of two, and one added to the denominator: scores of zero share it with the added one
    q, v = np.zeros((3, 1, 2)), np.array([[[3.0]], [[6.0]], [[12.0]]])
    assert plain.softmax_attention(q, np.zeros((3, 1, 2)), v, 1.0, window=2)[:, 0, 0] == pytest.approx([3.0, 4.5, 9.0])
    assert plain.softmax_attention(q, np.zeros((3, 1, 2)), v, 1.0, unit_sink=True)[:, 0, 0] == pytest.approx([1.5, 3.0, 21.0 / 4])
    # the delta rule: a key written twice with full strength holds the second value alone; with half, halfway
    k = np.array([[[1.0, 0.0]], [[1.0, 0.0]]])
    v = np.array([[[2.0]], [[10.0]]])
    out, S = plain.delta_rule(k, k, v, np.ones((2, 1)), np.ones((2, 1)))
    assert out[:, 0, 0] == pytest.approx([2.0, 10.0]) and S[0, :, 0] == pytest.approx([10.0, 0.0])
    out, _ = plain.delta_rule(k, k, v, np.full((2, 1), 0.5), np.full((2, 1), 0.5))
    assert out[:, 0, 0] == pytest.approx([1.0, 0.5 * 1.0 + 0.5 * (10.0 - 0.5)])
    # what is not kept is written
    out, S = plain.forget_and_write(np.ones((2, 1, 1)), np.array([[[0.25]], [[0.5]]]), np.array([[[4.0]], [[8.0]]]))
    assert out[:, 0, 0] == pytest.approx([3.0, 5.5])
    # sigmoid scores as weights on the input
    ids, scores = plain.route(np.array([[0.0, 2.0, -1.0]]), np.eye(3), 2)
    assert list(ids[0]) == [1, 0] and scores[0] == pytest.approx([1 / (1 + math.exp(-2.0)), 0.5])
    config = {"embedding": {"scale": 2.0, "bigram": {"buckets": 5, "mul_prev": 3, "mul_cur": 4}}}
    w = {"embed": np.arange(6.0).reshape(6, 1), "bigram": 100.0 * np.arange(6.0).reshape(6, 1)}
    assert plain.embed(config, w, np.array([4, 1, 5]))[:, 0] == pytest.approx([8.0 + 500.0, 2.0 + 100.0 * ((12 + 4) % 5), 10.0 + 100.0 * ((3 + 20) % 5)])


def test_run_order_of_the_plain_model():
    assert plain.run_order(zh.A) == [(0, None, False), (1, 0, True), (2, 0, False), (1, 1, True), (2, 1, False), (1, 2, True),
                                     (2, 2, False), (3, None, False)]
    assert plain.run_order(zh.B) == [(i, None, False) for i in range(3)]
