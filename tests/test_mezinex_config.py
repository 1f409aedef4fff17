"""The Mezinex design without a GPU: its config reader and the errors it raises, the model spec it becomes (the order in
which layers run, caches and states of every pass, the embedding's state, tensor names), the plain implementation on
cases made by hand, and a random model folder."""

import copy
import json

import numpy as np
import pytest

from plain import mezinex as plain
from qwen25vl_lite.config import ConfigError, resolve_architecture
from qwen25vl_lite.config.mezinex_config import MezinexConfig
from qwen25vl_lite.models.decoder import DecoderModel
from tiny_mezinex import TINY, Z1, Z2, Z3, Z4, Z5, make_model_dir


def model_of(raw):
    arch = resolve_architecture(raw)
    return DecoderModel(arch.build_spec(arch.config_from_dict(raw)))


def test_config_reads_every_size_and_constant():
    cfg = MezinexConfig.from_dict(Z1)
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps, cfg.streams, cfg.logit_scale, cfg.num_hidden_layers) == (211, 96, 1e-5, 3, 0.7, 3)
    assert (cfg.loop.start, cfg.loop.stop, cfg.loop.times) == (0, 2, 3)
    assert (cfg.pairs.buckets, cfg.pairs.mul_prev, cfg.pairs.mul_cur) == (37, 5, 3)
    s, r, a = (layer.mixer for layer in cfg.layers)
    assert (s.heads, s.vdim, s.state, s.groups, s.norm_groups, s.conv) == (6, 16, 24, 3, 2, 4)
    assert (r.width, r.blocks, r.conv) == (60, 5, 2)
    assert (a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank, a.scale, a.rot.dims, a.rot.base) == (3, 20, 12, 28, 24, 20, 0.3, 12, 1000.0)
    assert [layer.mlp and layer.mlp.ff for layer in cfg.layers] == [40, None, 56]
    bare = MezinexConfig.from_dict(Z5)
    assert bare.streams is None and bare.logit_scale == 1.0 and bare.loop is None
    assert MezinexConfig.from_dict(Z3).pairs is None


@pytest.mark.parametrize("path", [("vocab",), ("width",), ("norm",), ("norm", "eps"), ("layers", 0, "mixer", "state"), ("layers", 0, "mixer", "norm_groups"),
                                  ("layers", 0, "mixer", "conv"), ("layers", 0, "type"), ("layers", 0, "mlp", "ff"), ("layers", 1, "mixer", "blocks"),
                                  ("layers", 2, "mixer", "q_rank"), ("layers", 2, "mixer", "scale"), ("layers", 2, "mixer", "rot", "base"),
                                  ("loop", "times"), ("embedding", "bigram", "mul_cur")])
def test_a_missing_key_is_named(path):
    raw = copy.deepcopy(Z1)
    d = raw
    for key in path[:-1]:
        d = d[key]
    del d[path[-1]]
    with pytest.raises(ConfigError, match=str(path[-1])):
        MezinexConfig.from_dict(raw)


def test_config_errors():
    def broken(edit, message):
        raw = copy.deepcopy(Z1)
        edit(raw)
        with pytest.raises(ConfigError, match=message):
            MezinexConfig.from_dict(raw)

    broken(lambda r: r["layers"][0].update(type="convolution"), "unknown type")
    broken(lambda r: r["layers"][0]["mlp"].update(kind="sparse"), "unknown kind")
    broken(lambda r: r["layers"][0]["mixer"].update(groups=4), "groups")
    broken(lambda r: r["layers"][0]["mixer"].update(norm_groups=7), "equal parts")
    broken(lambda r: r["layers"][1]["mixer"].update(blocks=7), "blocks")
    broken(lambda r: r["layers"][2]["mixer"]["rot"].update(dims=14), "rot.dims")
    broken(lambda r: r["loop"].update(stop=4), "loop")
    broken(lambda r: r["loop"].update(times=0), "loop")
    broken(lambda r: r.update(streams=0), "streams")
    broken(lambda r: r["embedding"]["bigram"].update(buckets=0), "buckets")


def test_layers_run_in_the_looped_order_with_needs_of_their_own():
    model = model_of(Z1)
    assert [s.layer for s in model.spec.schedule] == [0, 1, 0, 1, 0, 1, 2] == plain.layer_order(Z1)
    assert len(model.blocks) == 3
    needs = model.stop_needs()
    for stop in (0, 2, 4):         # S [6, 24, 16], then three inputs of a convolution over 96 + 2 * 3 * 24 channels
        assert needs[stop].cache is None and needs[stop].state.shape == (6 * 24 * 16 + 3 * 240,) and needs[stop].state.dtype == "float32"
    for stop in (1, 3, 5):
        assert needs[stop].cache is None and needs[stop].state.shape == (2, 60)
    c = needs[6].cache
    assert (c.kv_heads, c.head_dim, c.v_dim, c.value_in_key, c.window) == (1, 36, 24, True, None) and needs[6].state is None
    for raw in (Z2, Z3, Z4, Z5):
        assert [s.layer for s in model_of(raw).spec.schedule] == plain.layer_order(raw)
    assert plain.layer_order(Z3) == [0, 1, 1, 2] and plain.layer_order(Z4) == [0, 1, 2, 0, 1, 2]


def test_the_embedding_asks_for_a_slot_of_its_own():
    from qwen25vl_lite.cache.manager import CacheManager

    model = model_of(Z1)
    other = model.other_state_needs()
    assert other["embedding"].shape == () and other["embedding"].dtype == "int32"
    assert model_of(Z3).other_state_needs() == {}
    manager = CacheManager(model.stop_needs(), num_pages=8, page_size=16, max_requests=2, other_states=other)
    manager.allocate_device("cpu", __import__("torch").float32)
    assert manager.states["embedding"].shape == (2,)
    manager.states["embedding"][:] = 9
    req = manager.open()
    assert int(manager.states["embedding"][req.slot]) == 0 and int(manager.states["embedding"].sum()) == 9
    manager.close(req)
    manager.check([])


def test_tensor_names_and_optional_tensors():
    names = model_of(Z1).expected_tensors()
    assert {"embed", "bigram", "final.norm", "head", "l0.norm1", "l0.norm2", "l0.hc1.in", "l0.hc1.out", "l0.hc2.mix", "l0.mix.in", "l0.mix.conv",
            "l0.mix.conv.b", "l0.mix.dt_bias", "l0.mix.A_log", "l0.mix.D", "l0.mix.norm", "l0.mix.o", "l0.mlp.gate", "l0.mlp.up", "l0.mlp.down",
            "l1.mix.y", "l1.mix.y.b", "l1.mix.ra", "l1.mix.ri.b", "l1.mix.lam", "l2.mix.dq", "l2.mix.dq.norm", "l2.mix.uq", "l2.mix.dkv",
            "l2.mix.dkv.norm", "l2.mix.uk", "l2.mix.uv", "l2.mix.g", "l2.mix.o"} <= set(names)
    assert names["bigram"].shape == (38, 96) and names["l0.mix.in"].shape == (96 + 240 + 6, 96) and names["l0.mix.conv"].shape == (240, 4)
    assert names["l2.mix.uq"].shape == (3 * 32, 20) and names["l2.mix.dkv"].shape == (36, 96) and names["l0.hc1.mix"].shape == (3, 3)
    required = {n for n, ts in names.items() if not ts.optional}
    assert {"l1.norm2", "l1.hc2.in", "l1.hc2.mix"} & required == set() and "l1.mlp.gate" not in names      # no feed-forward there
    assert "l2.mix.sink" not in names and "l2.mix.q" not in names
    assert not any(".hc" in n for n in model_of(Z5).expected_tensors()) and "bigram" not in model_of(Z3).expected_tensors()


def test_plain_pair_rows_by_hand():
    assert plain.bigram_rows([4, 2, 2, 9], 10, 3, 7) == [10, (4 * 3 + 2 * 7) % 10, (2 * 3 + 2 * 7) % 10, (2 * 3 + 9 * 7) % 10]


def test_plain_stream_by_hand():
    """[from, to]: with mix[0, 1] alone the second row becomes the first, and the first nothing but the result."""
    streams = np.array([[[1.0, 2.0]], [[5.0, 7.0]]])
    assert np.allclose(plain.hyper_read(streams, np.array([2.0, -1.0])), [[-3.0, -3.0]])
    mix = np.array([[0.0, 1.0], [0.0, 0.0]])
    new = plain.hyper_write(streams, mix, np.array([10.0, 0.0]), np.array([[1.0, 1.0]]))
    assert np.allclose(new, [[[10.0, 10.0]], [[1.0, 2.0]]])


def test_plain_state_space_by_hand():
    """Two steps of a state of one row and one column, and the direct sum over the past for larger ones."""
    one = lambda *v: np.array(v, dtype=np.float64).reshape(len(v), 1, 1)
    dt = np.array([[0.5], [2.0]])
    y = plain.state_space(one(3.0, 4.0), one(1.0, 0.5), one(2.0, 1.0), dt, np.array([0.0]), np.array([0.1]))
    s1 = 0.5 * 1.0 * 3.0
    s2 = np.exp(-2.0) * s1 + 2.0 * 0.5 * 4.0
    assert np.allclose(y.reshape(-1), [2.0 * s1 + 0.3, s2 + 0.4])
    rng = np.random.default_rng(0)
    T, H, V, G, N = 9, 4, 3, 2, 5
    x, b, c = rng.standard_normal((T, H, V)), rng.standard_normal((T, G, N)), rng.standard_normal((T, G, N))
    dt, a_log, d = rng.uniform(0.01, 1.0, (T, H)), rng.uniform(-2, 1, H), rng.standard_normal(H)
    y = plain.state_space(x, b, c, dt, a_log, d)
    total = np.cumsum(-np.exp(a_log) * dt, axis=0)
    for h in range(H):
        for t in range(T):
            want = d[h] * x[t, h] + sum(np.exp(total[t, h] - total[j, h]) * dt[j, h] * (c[t, h // 2] @ b[j, h // 2]) * x[j, h] for j in range(t + 1))
            assert np.allclose(y[t, h], want)


def test_plain_convolution_and_recurrence_by_hand():
    x = np.array([[1.0], [10.0], [100.0]])
    assert np.allclose(plain.causal_conv(x, np.array([[3.0, 2.0, 1.0]]), np.array([0.5])), [[1.5], [12.5], [123.5]])
    u, r, i = np.array([[2.0], [1.0]]), np.array([[0.25], [1.0]]), np.array([[1.0], [0.5]])
    lam = np.array([np.log(np.expm1(0.125))])                     # softplus(lam) = 1/8, so log a = -r
    s = plain.linear_recurrence(u, r, i, lam)
    a0, a1 = np.exp(-0.25), np.exp(-1.0)
    s0 = np.sqrt(1 - a0 ** 2) * 2.0                               # no special case for the first token
    assert np.allclose(s.reshape(-1), [s0, a1 * s0 + np.sqrt(1 - a1 ** 2) * 0.5])


@pytest.mark.parametrize("name", sorted(TINY))
def test_random_model_folder_loads_into_the_plain_implementation(tmp_path, name):
    folder = make_model_dir(tmp_path, name, "bfloat16")
    cfg, w = plain.load_model_dir(folder)
    assert set(w) == {n for n, ts in model_of(TINY[name][0]).expected_tensors().items() if not ts.optional}
    streams = []
    logits = plain.forward(cfg, w, [1, 2, 3, 4, 5], streams)
    assert logits.shape == (5, cfg["vocab"]) and np.isfinite(logits).all() and len(streams) == len(plain.layer_order(cfg))


def test_command_line_writes_a_random_model_of_the_design(tmp_path):
    from qwen25vl_lite import cli
    from qwen25vl_lite.config import known_architectures

    assert "Mezinex" in known_architectures()
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(Z3))
    out = tmp_path / "model"
    assert cli.main(["random-model", "--config", str(cfg), "--out", str(out), "--seed", "4"]) == 0
    config, w = plain.load_model_dir(str(out))
    assert config["architecture"] == "Mezinex" and np.isfinite(plain.forward_logits(config, w, [1, 2, 3])).all()
