"""The Sudilorn design without a GPU: its config reader and the errors it raises, the model spec it becomes (caches and states
of every layer, tensor names, constants that are folded together), the delta rule's work lists, the plain implementation on
cases made by hand, and a random model folder."""

import copy
import json

import numpy as np
import pytest

from plain import sudilorn as plain
from qwen25vl_lite.config import ConfigError, resolve_architecture
from qwen25vl_lite.config.sudilorn_config import SudilornConfig
from qwen25vl_lite.models.decoder import DecoderModel
from qwen25vl_lite.ops import delta_rule
from tiny_sudilorn import TINY, Z1, Z2, Z3, Z4, Z5, make_model_dir


def model_of(raw):
    arch = resolve_architecture(raw)
    return DecoderModel(arch.build_spec(arch.config_from_dict(raw)))


def test_config_reads_every_size_and_constant():
    cfg = SudilornConfig.from_dict(Z1)
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps, cfg.residual_mult, cfg.num_hidden_layers) == (211, 96, 1e-5, 0.7, 2)
    p, a = (layer.mixer for layer in cfg.layers)
    l, r = p.left, p.right
    assert (l.heads, l.kv_heads, l.dim, l.vdim, l.scale, l.window, l.keep_first, l.rot.dims, l.rot.base, l.rot.scaling) == (6, 2, 24, 20, 0.3, 9, 3, 10, 500.0, None)
    assert (r.heads, r.kv_heads, r.dim, r.vdim, r.conv, p.left_scale, p.right_scale) == (4, 2, 20, 24, 2, 0.7, 1.3)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.conv, a.diff, a.scale, a.window, a.rot.dims) == (6, 3, 20, 28, 3, 0.35, 0.3, 17, 12)
    assert a.rot.scaling_dict() == {"kind": "ramp", "factor": 2.0, "original": 64.0, "fast": 8.0, "slow": 1.0}
    f = cfg.layers[0].mlp
    assert (f.experts, f.top, f.ff, f.groups, f.keep) == (10, 3, 40, 5, 2) and cfg.layers[1].mlp is None
    bare = SudilornConfig.from_dict(Z3)
    assert bare.layers[0].mixer.left.kv_heads == 1 and bare.layers[0].mixer.left.rot is None and bare.layers[1].mixer.window is None
    assert (bare.layers[1].mlp.groups, bare.layers[1].mlp.keep) == (1, 1)


@pytest.mark.parametrize("path", [("vocab",), ("width",), ("norm",), ("norm", "eps"), ("layers",), ("layers", 0, "type"), ("layers", 0, "mixer", "left"),
                                  ("layers", 0, "mixer", "left", "scale"), ("layers", 0, "mixer", "left", "dim"), ("layers", 0, "mixer", "left", "rot", "base"),
                                  ("layers", 0, "mixer", "right", "conv"), ("layers", 0, "mixer", "right", "vdim"), ("layers", 0, "mlp", "expert"),
                                  ("layers", 0, "mlp", "router", "top"), ("layers", 1, "mixer", "diff"), ("layers", 1, "mixer", "heads"),
                                  ("layers", 1, "mixer", "rot", "scaling", "slow")])
def test_a_missing_key_is_named(path):
    raw = copy.deepcopy(Z1)
    d = raw
    for key in path[:-1]:
        d = d[key]
    del d[path[-1]]
    with pytest.raises(ConfigError, match=str(path[-1])):
        SudilornConfig.from_dict(raw)


def test_config_errors():
    def broken(edit, message):
        raw = copy.deepcopy(Z1)
        edit(raw)
        with pytest.raises(ConfigError, match=message):
            SudilornConfig.from_dict(raw)

    broken(lambda r: r["layers"][0].update(type="convolution"), "unknown type")
    broken(lambda r: r["layers"][0]["mlp"].update(kind="dense"), "unknown kind")
    broken(lambda r: r["layers"][0]["mixer"]["left"].update(kv_heads=4), "kv_heads")
    broken(lambda r: r["layers"][0]["mixer"]["right"].update(conv=17), "conv")
    broken(lambda r: r["layers"][1]["mixer"]["rot"].update(dims=22), "rot.dims")
    broken(lambda r: r["layers"][0]["mlp"]["router"]["groups"].update(count=3), "equal groups")
    broken(lambda r: r["layers"][0]["mlp"]["router"].update(top=5), "choices")
    broken(lambda r: r["layers"][0]["mixer"]["left"]["mask"].update(size=-1), "mask.size")


def test_caches_and_states_of_every_layer():
    needs = model_of(Z1).stop_needs()
    c = needs[0].cache
    assert (c.kv_heads, c.head_dim, c.v_dim, c.window, c.keep_first) == (2, 24, 20, 9, 3)
    # S [4, 20, 24], then one input of a convolution over 2 * 2 * 20 + 4 * 24 channels
    assert needs[0].state.shape == (4 * 20 * 24 + 176,) and needs[0].state.dtype == "float32"
    c = needs[1].cache                                  # both maps' keys side by side over one value
    assert (c.kv_heads, c.head_dim, c.v_dim, c.window, c.keep_first) == (3, 40, 28, 17, 0)
    assert needs[1].state.shape == (2 * (2 * 6 * 20 + 2 * 3 * 20 + 3 * 28),)
    n3 = model_of(Z3).stop_needs()
    assert n3[1].state is None and n3[1].cache.window is None           # one tap carries nothing
    assert n3[0].state.shape == (92,)                   # 13 * 7 floats, filled up to a multiple of four
    for raw in (Z2, Z4, Z5):
        assert all(n.cache is not None and n.state is not None for n in model_of(raw).stop_needs())


def test_tensor_names_and_optional_tensors():
    names = model_of(Z1).expected_tensors()
    assert {"embed", "final.norm", "head", "l0.norm1", "l0.norm2", "l0.ls1", "l0.ls2", "l0.mix.left.q", "l0.mix.left.q.b", "l0.mix.left.o", "l0.mix.right.q",
            "l0.mix.right.q.conv", "l0.mix.right.b", "l0.mix.right.A_log", "l0.mix.right.norm", "l0.mix.right.a", "l0.mix.right.dt_bias", "l0.mix.right.g",
            "l0.mix.right.o", "l0.mlp.e9.up", "l0.mlp.e0.down", "l0.mlp.router", "l0.mlp.correction", "l1.mix.q", "l1.mix.q.norm", "l1.mix.k.conv", "l1.mix.v.conv",
            "l1.mix.lq1", "l1.mix.lk2", "l1.mix.g", "l1.mix.o"} <= set(names)
    assert names["l1.mix.q"].shape == (240, 96) and names["l1.mix.k"].shape == (120, 96) and names["l1.mix.g"].shape == (168, 96)
    assert names["l0.mix.right.v.conv"].shape == (96, 2) and names["l0.mix.right.b"].shape == (4, 96) and names["l0.mlp.router"].shape == (10, 96)
    required = {n for n, ts in names.items() if not ts.optional}
    assert {"l1.norm2", "l1.ls2"} & required == set() and "l1.mlp.router" not in names       # no feed-forward there
    assert not any(n.endswith(("left.o.b", "left.sink", "gate")) for n in names)


def test_constants_that_are_folded_together():
    spec = model_of(Z1).spec
    assert [n.params["gain"] for n in spec.layers[0].norms if n.kind == "channel_scale"] == [pytest.approx(0.7 * 0.7), pytest.approx(0.7)]
    assert [b[2] for b in spec.layers[0].mixer.params["branches"]] == [1.0, pytest.approx(1.3 / 0.7)]
    zero = model_of(Z3).spec.layers[0]                  # a left branch of weight 0 cannot be divided by
    assert [b[2] for b in zero.mixer.params["branches"]] == [0.0, 1.0] and zero.norms[1].params["gain"] == 1.0


def test_work_lists_of_the_delta_rule():
    p = delta_rule.plan([1, 200, 15, 16, 64], True)
    assert p["chunks"].reshape(-1, 2).tolist() == [[1, 65], [65, 129], [129, 193], [193, 201], [216, 232], [232, 296]]
    assert p["runs"].reshape(-1, 4).tolist() == [[1, 201, 1, 0], [216, 232, 3, 4], [232, 296, 4, 5]]
    assert p["walked"].reshape(-1, 3).tolist() == [[0, 1, 0], [201, 216, 2]]
    for p in (delta_rule.plan([1, 1, 9], True), delta_rule.plan([1, 200, 15], False)):
        assert all(a.size == 0 for a in p.values())     # all entries are walked


# ---- the plain implementation by hand ------------------------------------------------------------------------


def test_plain_masks_by_hand():
    seen = plain.visible(7, {"size": 2, "keep_first": 2})
    assert seen[5].tolist() == [True, True, False, False, True, True, False] and seen[1].tolist() == [True, True] + [False] * 5
    assert plain.visible(4, {"size": 1}).tolist() == np.eye(4, dtype=bool).tolist()
    assert plain.visible(3, None).tolist() == np.tril(np.ones((3, 3), dtype=bool)).tolist()


def test_plain_rotation_by_hand():
    x = np.zeros((2, 1, 6))
    x[1, 0] = [1.0, 2.0, 3.0, 4.0, 5.0, 6.0]
    c, s = np.cos(1.0), np.sin(1.0)
    c2, s2 = np.cos(0.1), np.sin(0.1)
    rot = {"dims": 4, "base": 100.0}
    assert np.allclose(plain.rotate(x, rot, "halves")[1, 0], [c - 3 * s, 2 * c2 - 4 * s2, 3 * c + s, 4 * c2 + 2 * s2, 5, 6])
    assert np.allclose(plain.rotate(x, rot, "pairs")[1, 0], [c - 2 * s, 2 * c + s, 3 * c2 - 4 * s2, 4 * c2 + 3 * s2, 5, 6])
    f, mag = plain.ramp_frequencies(8, 100.0, {"factor": 4.0, "original": 2.0 * np.pi * 10.0, "fast": 10.0, "slow": 1.0})
    # fast: the pair that turns ten times, number 0; slow: the one that turns once, number 8 ln 10 / (2 ln 100) = 2
    assert mag == pytest.approx(0.1 * np.log(4.0) + 1.0)
    assert np.allclose(f / 100.0 ** (-np.arange(4) / 4.0), [1.0, 0.5 + 0.5 / 4.0, 0.25, 0.25])


def test_plain_delta_rule_by_hand():
    """Writing along a key replaces what the key answered (strength 1), and leaves orthogonal keys alone; the read-out sees
    the token's own write; the decay comes before the difference is taken."""
    e = np.eye(2)
    q = k = np.array([e[0], e[1], e[0]])[:, None]
    v = np.array([[[3.0]], [[5.0]], [[7.0]]])
    one = np.ones((3, 1))
    o, S = plain.delta_rule(q, k, v, one, one)
    assert np.allclose(o.reshape(-1), [3, 5, 7]) and np.allclose(S.reshape(-1), [7, 5])
    o, S = plain.delta_rule(q, k, v, 0.5 * one, 0.5 * one)
    s0 = 0.5 * (0.5 * 1.5)
    assert np.allclose(o.reshape(-1), [1.5, 2.5, s0 + 0.5 * (7 - s0)])
    assert np.allclose(plain.unit_vectors(np.array([3e-4, 4e-4])), np.array([3e-4, 4e-4]) / np.sqrt(25e-8 + 1e-6))


def test_plain_differential_pieces_by_hand():
    t = {n: np.array(v) for n, v in dict(lq1=[1.0, 2.0], lk1=[0.5, 0.25], lq2=[1.0, 0.0], lk2=[-1.0, 9.0]).items()}
    assert plain.mixing_weight(t, 0.3) == pytest.approx(np.exp(1.0) - np.exp(-1.0) + 0.3)
    o = plain.differential_heads(np.array([4.0, 2.0]), np.array([2.0, 0.0]), 0.5, 0.2, 0.0)
    assert np.allclose(o, 0.8 * np.array([3.0, 2.0]) / np.sqrt(6.5))


def test_plain_router_by_hand():
    """A group's mark is the sum of its two largest numbers, corrections count in the choice and not in the weights, and
    experts of other groups lose even against negative numbers."""
    logit = lambda p: np.log(np.array(p) / (1 - np.array(p)))
    r = {"experts": 6, "top": 2, "groups": {"count": 2, "keep": 1}}
    z = logit([0.9, 0.1, 0.1, 0.6, 0.5, 0.1])          # group 0: 1.0 with the largest number, group 1: 1.1
    chosen, w = plain.route(z, np.zeros(6), r)
    assert chosen.tolist() == [3, 4] and np.allclose(w, [0.6, 0.5])
    chosen, w = plain.route(z, np.array([-2.0, -2.0, -2.0, -3.0, -3.0, -3.0]), r)
    assert chosen.tolist() == [0, 1] and np.allclose(w, [0.9, 0.1])
    chosen, w = plain.route(z, np.array([0, 0, 0, 0, 0, 0.9]), r)
    assert chosen.tolist() == [5, 3] and np.allclose(w, [0.1, 0.6])


@pytest.mark.parametrize("name", sorted(TINY))
def test_random_model_folder_loads_into_the_plain_implementation(tmp_path, name):
    folder = make_model_dir(tmp_path, name, "bfloat16")
    cfg, w = plain.load_model_dir(folder)
    assert set(w) == {n for n, ts in model_of(TINY[name][0]).expected_tensors().items() if not ts.optional}
    after = []
    logits = plain.forward(cfg, w, [1, 2, 3, 4, 5], after)
    assert logits.shape == (5, cfg["vocab"]) and np.isfinite(logits).all() and len(after) == len(cfg["layers"])


def test_command_line_writes_a_random_model_of_the_design(tmp_path):
    from qwen25vl_lite import cli
    from qwen25vl_lite.config import known_architectures

    assert "Sudilorn" in known_architectures()
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(Z3))
    out = tmp_path / "model"
    assert cli.main(["random-model", "--config", str(cfg), "--out", str(out), "--seed", "4"]) == 0
    config, w = plain.load_model_dir(str(out))
    assert config["architecture"] == "Sudilorn" and np.isfinite(plain.forward_logits(config, w, [1, 2, 3])).all()
