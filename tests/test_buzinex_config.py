"""Buzinex's configuration and its place in the registries, and the plain implementation's pieces against direct
arithmetic (no GPU)."""
import copy
import math

import numpy as np
import pytest

import buzinex_helpers as bh
import helpers
import plain_buzinex as plain
from sprout_lm_b200.config import BuzinexConfig, ConfigError, parse_config, registered_architectures
from sprout_lm_b200.config.specs import LayerSpec, PartSpec
from sprout_lm_b200.models.decoder import DecoderModel
from sprout_lm_b200.parts import build_block, build_part


def test_registered_and_round_trip():
    assert "Buzinex" in registered_architectures()
    for raw, _, _ in bh.CONFIGS.values():
        config = parse_config(raw)
        assert isinstance(config, BuzinexConfig)
        assert parse_config(config.to_dict()) == config and config.to_dict() == raw


def test_model_spec_follows_the_file():
    spec = parse_config(bh.A).model_spec()
    assert [layer.block for layer in spec.layers] == ["sandwich_norm"] * 5
    assert [layer.mixer.kind for layer in spec.layers] == ["latent_attention", "rwkv_time_mixing", "multimap_attention",
                                                          "latent_attention", "rwkv_time_mixing"]
    assert [layer.feed_forward.kind for layer in spec.layers] == ["gated_mlp", "gated_mlp", "none", "none", "none"]
    assert [len(layer.norms) for layer in spec.layers] == [4, 4, 2, 2, 2]
    assert all(norm.kind == "rmsnorm" for layer in spec.layers for norm in layer.norms)
    latent, full = spec.layers[0].mixer.params, spec.layers[2].mixer.params
    assert latent["window"] == 5 and latent["position"].kind == "rope_interleaved" and latent["position"].params["dims"] == 6
    assert latent["scale"] == 0.31 and "q_rank" not in latent
    assert full["softcap"] == 7.0 and full["query_growth"] == (0.9, 3) and full["position"].kind == "none" and full["qk_norm_eps"] == 1e-5
    assert spec.head.params["tied_to"] == "embed" and spec.head.params["scale"] == 0.6 and spec.head.params["softcap"] == 11.0
    assert spec.embedding.params["scale"] == 3.0
    assert [(c.layer, c.cache) for c in spec.order] == [(i, i) for i in range(5)]
    model = DecoderModel(spec)
    caches = model.cache_specs()
    assert (caches[0].kind, caches[0].window, caches[0].head_dim, caches[0].value_dim) == ("window", 5, 26, 0)
    assert caches[1] is None and caches[4] is None and caches[3].window == 19
    assert (caches[2].kind, caches[2].kv_heads, caches[2].head_dim, caches[2].value_dim) == ("full", 3, 9, 11)
    states = model.state_specs()
    assert [s.shape for s in states[1]] == [(36,), (3, 6, 6)] and [s.shape for s in states[4]] == [(36,), (2, 11, 11)]
    assert states[0] is None and states[-1] is None
    names = {decl.name: decl.shape for decl in model.tensor_decls()}
    assert names["embed"] == (211, 36) and "head" not in names and names["final.norm"] == (36,)
    assert names["l0.norm1b"] == names["l0.norm2b"] == (36,) and "l2.norm2" not in names and names["l2.norm1b"] == (36,)
    assert names["l0.mix.q"] == (48, 36) and names["l0.mix.dkv"] == (26, 36) and names["l0.mix.dkv.norm"] == (20,)
    assert names["l0.mix.uk"] == (30, 20) and names["l0.mix.uv"] == (21, 20) and names["l0.mix.sink"] == (3,) and names["l0.mix.o"] == (36, 21)
    assert names["l2.mix.q"] == (54, 36) and names["l2.mix.k"] == (27, 36) and names["l2.mix.v"] == (33, 36) and names["l2.mix.q.norm"] == (9,)
    assert names["l1.mix.mu.r"] == names["l1.mix.mu.w"] == (36,) and names["l1.mix.g"] == (18, 36) and names["l1.mix.u"] == (3, 6)
    assert names["l1.mix.w1"] == (5, 36) and names["l1.mix.w2"] == (18, 5) and names["l1.mix.w0"] == names["l1.mix.norm"] == (18,)
    assert names["l1.mlp.gate"] == (20, 36) and names["l1.mlp.down"] == (36, 20)


def test_inner_size_of_the_decay_comes_from_the_tensors():
    raw = copy.deepcopy(bh.A)
    del raw["layers"][1]["mixer"]["rank"]
    names = {decl.name: decl.shape for decl in DecoderModel(parse_config(raw).model_spec()).tensor_decls()}
    assert names["l1.mix.w1"] == (None, 36) and names["l1.mix.w2"] == (18, None)
    assert parse_config(raw).to_dict() == raw


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][2]["mixer"].__setitem__("heads", 5), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 4), "rot.dims"),
    (lambda c: (c["layers"][0]["mixer"]["rot"].__setitem__("dims", 7), c["layers"][0]["mixer"].__setitem__("rot_dim", 7)), "even"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("base", 1.0), "base"),
    (lambda c: c["layers"][0]["mixer"].pop("mask"), "mask"),
    (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "size"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_rank", 2000), "at most 1024"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("scale", 0), "scale"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("vdim", 600), "at most 512"),
    (lambda c: c["layers"][2]["mixer"].pop("softcap"), "softcap"),
    (lambda c: c["layers"][2]["mixer"].pop("q_temp"), "q_temp"),
    (lambda c: c["layers"][2]["mixer"]["q_temp"].__setitem__("every", 0), "every"),
    (lambda c: c["layers"][2]["mixer"]["q_temp"].pop("coef"), "coef"),
    (lambda c: c["layers"][1]["mixer"].pop("dim"), "dim"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("rank", 0), "rank"),
    (lambda c: c["layers"][1].__setitem__("type", "rwkv"), "type"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "kind"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("ff", -1), "ff"),
    (lambda c: c.pop("logit_scale"), "logit_scale"),
    (lambda c: c.__setitem__("logit_softcap", 0), "logit_softcap"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c["norm"].__setitem__("eps", 0), "eps"),
    (lambda c: c.__setitem__("layers", []), "layers"),
    (lambda c: c.__setitem__("vocab", 0), "vocab"),
])
def test_refusals(edit, text):
    raw = copy.deepcopy(bh.A)
    edit(raw)
    with pytest.raises(ConfigError, match=text):
        parse_config(raw)


def test_parts_refuse_what_they_cannot_compute():
    base = {"hidden_size": 16, "heads": 2, "kv_heads": 1, "dim": 4, "value_dim": 4, "scale": 1.0, "position": PartSpec("none", {}), "maps": 1}
    build_part("mixer", PartSpec("multimap_attention", {**base, "query_growth": (0.1, 4)}))
    for wrong in ((0.1, 0), (0.1, 2.5)):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("multimap_attention", {**base, "query_growth": wrong}))
    latent = {"hidden_size": 16, "heads": 2, "dim": 4, "rot_dim": 0, "value_dim": 4, "kv_rank": 8, "scale": 1.0, "eps": 1e-5,
              "position": PartSpec("none", {})}
    assert build_part("mixer", PartSpec("latent_attention", latent)).cache_spec().kind == "full"
    for wrong in ({"window": 0}, {"scale": 0.0}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("latent_attention", {**latent, **wrong}))
    for wrong in ({"dim": 0}, {"decay_rank": 0}, {"eps": 0.0}):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("rwkv_time_mixing", {"hidden_size": 16, "heads": 2, "dim": 4, "eps": 1e-5, **wrong}))
    mixer = PartSpec("rwkv_time_mixing", {"hidden_size": 16, "heads": 2, "dim": 4, "eps": 1e-5})
    norms = tuple(PartSpec(kind, {"size": 16, "eps": 1e-5, "name": f"n{i}"}) for i, kind in enumerate(("rmsnorm", "layernorm")))
    with pytest.raises(ValueError):
        build_block(LayerSpec("sandwich_norm", "", mixer, PartSpec("none", {}), norms))


def test_a_lost_state_a_dropped_sink_or_a_shifted_window_shows(tmp_path):
    """The test models are made so that each mechanism matters: a mistake planted in the plain implementation moves the logits
    by far more than the bar."""
    directory = bh.make_model_dir(tmp_path, "A")
    tokens = helpers.random_tokens(np.random.default_rng(31), 60, bh.A["vocab"])
    full = bh.plain_logits(directory, tokens)
    bar = 0.15

    def moved(other, places=slice(None)):
        """The largest change at any place: a fault is found if one place is over the bar."""
        return max(bh.relative(a, b) for a, b in zip(other, full[places]))
    assert moved(bh.plain_logits(directory, tokens[30:]), slice(30, None)) > bar
    config, tensors = bh.plain_model(directory)
    for label, change in {
            "sinks": lambda k, v: np.full_like(v, -1e9) if k.endswith(".sink") else v,
            "bonus": lambda k, v: np.zeros_like(v) if k.endswith(".u") else v,
            "blends": lambda k, v: np.zeros_like(v) if ".mu." in k else v,
            "swapped blends": lambda k, v: tensors[k.replace(".mu.k", ".mu.v")] if k.endswith(".mu.k") else v,
            "decay offsets": lambda k, v: v + 0.7 if k.endswith(".w0") else v,
            "decay from the input": lambda k, v: np.zeros_like(v) if k.endswith(".w2") else v,
            "query norm": lambda k, v: np.ones_like(v) if k.endswith(".q.norm") else v,
            "key norm": lambda k, v: np.ones_like(v) if k.endswith(".k.norm") else v,
            "latent norm": lambda k, v: np.ones_like(v) if k.endswith(".dkv.norm") else v,
            "heads' norm": lambda k, v: np.ones_like(v) if k.endswith(".mix.norm") else v,
            "norm after": lambda k, v: np.ones_like(v) if k.endswith("norm1b") else v}.items():
        assert moved(plain.forward(config, {k: change(k, v) for k, v in tensors.items()}, tokens)) > bar, label
    edits = [lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", 6),
             lambda c: c["layers"][3]["mixer"]["mask"].__setitem__("size", 18),
             lambda c: c["layers"][3]["mixer"]["mask"].__setitem__("size", 20),
             lambda c: c["layers"][3]["mixer"]["rot"].__setitem__("base", 300.0),
             lambda c: c["layers"][2]["mixer"]["q_temp"].__setitem__("coef", 0.0),
             lambda c: c["layers"][2]["mixer"]["q_temp"].__setitem__("every", 9),
             lambda c: c["layers"][2]["mixer"].__setitem__("softcap", 40.0),
             lambda c: c["layers"][1].__setitem__("mlp", None),
             lambda c: c["embedding"].__setitem__("scale", 1.0),
             lambda c: c.__setitem__("logit_scale", 1.0),
             lambda c: c.__setitem__("logit_softcap", 2.0)]
    for number, edit in enumerate(edits):
        changed = copy.deepcopy(config)
        edit(changed)
        assert moved(plain.forward(changed, tensors, tokens)) > bar, number
    # pieces of the mechanisms left out
    real = {key: getattr(plain, key) for key in ("rotate_pairs", "decay_with_bonus", "blend_with_before", "latent_scores", "query_growth")}

    def planted(key, fn):
        try:
            setattr(plain, key, fn)
            return moved(plain.forward(config, tensors, tokens))
        finally:
            setattr(plain, key, real[key])
    half = lambda x, p, b: np.concatenate(np.split(real["rotate_pairs"](np.stack(np.split(x, 2, -1), -1).reshape(x.shape), p, b)
                                                   .reshape(*x.shape[:-1], -1, 2), 2, -1), -2)[..., 0]
    assert planted("rotate_pairs", half) > bar                                            # pairs (i, i + half) instead
    assert planted("decay_with_bonus", lambda r, k, v, w, u: real["decay_with_bonus"](r, k, v, w, np.ones_like(u))) > bar
    assert planted("decay_with_bonus", lambda r, k, v, w, u: real["decay_with_bonus"](r, k, v, np.minimum(w, 0.9), u)) > bar
    assert planted("blend_with_before", lambda h, mu: real["blend_with_before"](h, mu, before=h[0])) > bar
    assert planted("latent_scores", lambda a, b, c, d, s: real["latent_scores"](a, 0 * b, c, d, s)) > bar
    # a step of the growth one position late touches few queries: the 32-bit runs find it
    assert planted("query_growth", lambda p, c, e: real["query_growth"](np.asarray(p) - 1, c, e)) > 0.01


# ------------------------------------------------------------------------------------------------ the plain pieces
def test_plain_pieces_against_direct_arithmetic():
    x = np.array([[[1.0, 2.0, 3.0, 4.0]]])
    assert plain.rotate_pairs(x, np.array([np.pi / 2]), 1e12)[0, 0] == pytest.approx([-2.0, 1.0, 3.0, 4.0], abs=1e-5)
    second = plain.rotate_pairs(x, np.array([5]), 100.0)[0, 0]
    assert second[2:] == pytest.approx([3 * math.cos(0.5) - 4 * math.sin(0.5), 4 * math.cos(0.5) + 3 * math.sin(0.5)])
    weights = plain.softmax_rows(np.array([[0.0, -np.inf, 0.0]]), sink=math.log(2.0))
    assert weights[0] == pytest.approx([0.25, 0.0, 0.25])
    assert plain.softmax_rows(np.array([[3.0, 3.0]]))[0] == pytest.approx([0.5, 0.5])
    assert plain.visible(4, 2).astype(int).tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    assert plain.query_growth([0, 1, 2, 3, 6], 0.5, 3) == pytest.approx([1.0, 1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2),
                                                                        1 + 0.5 * math.log(3)])
    h = np.array([[4.0], [8.0], [0.0]])
    assert plain.blend_with_before(h, np.array([0.25]))[:, 0] == pytest.approx([3.0, 7.0, 2.0])
    assert plain.blend_with_before(h[1:], np.array([0.25]), before=h[0])[:, 0] == pytest.approx([7.0, 2.0])
    # the bonus weighs the current token only; the decay touches what was there before, not the write
    one = np.ones((3, 1, 1))
    out, S = plain.decay_with_bonus(one, one, np.array([2.0, 4.0, 8.0]).reshape(3, 1, 1), 0.5 * one, np.array([[3.0]]))
    assert out[:, 0, 0] == pytest.approx([6.0, 2.0 + 12.0, 5.0 + 24.0]) and S[0, 0, 0] == pytest.approx(10.5)
    assert plain.soft_cap(np.array([1e9, 0.0]), 7.0) == pytest.approx([7.0, 0.0])
    config = {"norm": {"eps": 1e-12}, "logit_scale": 0.5, "logit_softcap": 3.0}
    w = {"final.norm": np.array([2.0, 1.0]), "embed": np.array([[1.0, 0.0], [1.0, 1.0]])}
    assert plain.head(config, w, np.array([[3.0, 3.0]]))[0] == pytest.approx([3 * math.tanh(1 / 3), 3 * math.tanh(0.5)])
