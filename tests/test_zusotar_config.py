"""The Zusotar configuration on the CPU: what is read, what is refused, the layout as parts, the tensor names, the cache,
what the parts do to their weights, and the plain implementation's own pieces against hand-made cases."""
import copy

import numpy as np
import pytest
import torch

import plain_zusotar as plain
import zusotar_cases as sc
from coheryn_ai_studio_b200.config import ConfigError, architecture_for
from coheryn_ai_studio_b200.config.zusotar import ZusotarConfig, zusotar_model_spec
from coheryn_ai_studio_b200.parts.base import FixedState, PagedKV, Runtime
from coheryn_ai_studio_b200.parts.model import DecoderModel

CPU = Runtime(torch.float32, torch.device("cpu"))


def model_of(cfg):
    return DecoderModel(zusotar_model_spec(ZusotarConfig.from_dict(cfg)), CPU)


def test_round_trip_and_registry():
    for cfg, _ in sc.CASES.values():
        c = ZusotarConfig.from_dict(cfg)
        assert ZusotarConfig.from_dict(c.to_dict()) == c
        assert architecture_for(cfg).name == "Zusotar"
        d = architecture_for(cfg).describe(c)
        assert d["context"] == cfg["max_positions"] and d["capabilities"]["fixed_state_bytes_per_request"] > 0


def test_layout_tensor_names_and_cache():
    m = model_of(sc.S1)
    specs = m.tensor_specs()
    assert {"embed", "pos", "head", "final.norm", "l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.dwa", "l4.dwa", "l0.mix.q",
            "l0.mix.dkv", "l0.mix.dkv.norm", "l0.mix.uk", "l0.mix.uv", "l0.mix.sink", "l0.mix.o", "l0.mlp.router", "l0.mlp.e7.down",
            "l0.mlp.shared.gate", "l1.mix.a1", "l1.mix.a2", "l1.mix.a2.b", "l1.mix.norm", "l1.mix.g", "l1.mlp.gate", "l1.mlp.down",
            "l2.mix.r1", "l2.mix.r2", "l2.mix.g", "l2.mix.v"} <= set(specs)
    assert not {"l0.mix.g", "l2.mix.sink", "l2.mlp.shared.gate", "l3.norm2", "l3.norm2b", "l3.mlp.gate", "l0.mlp.shared.sg",
                "l0.mlp.correction"} & set(specs)
    assert specs["pos"].shape == (320, 64) and specs["l0.mix.dkv"].shape == (48 + 16, 64) and specs["l2.mix.g"].shape == (4 * 16, 64)
    assert specs["l1.mix.a2"].shape == (2 * 32, 16) and specs["l1.mix.norm"].shape == (16,) and specs["l3.dwa"].shape == (5,)
    free = copy.deepcopy(sc.S1)
    del free["layers"][1]["mixer"]["a_rank"]          # a checkpoint's tensors give the rank
    assert model_of(free).tensor_specs()["l1.mix.a1"].shape == (-1, 64)
    assert [e.average for e in m.spec.schedule] == [f"l{i}.dwa" for i in range(5)]
    assert m.cache_requirements() == [PagedKV(1, 64, None, 0), FixedState((2 * 32 * 16,), torch.float32), PagedKV(2, 32, 24, 16),
                                      FixedState((4 * 16 * 32,), torch.float32), PagedKV(1, 16, 9, 32)]


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "conv"), (("layers", 2, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "rot", "dims"), 18),
    (("layers", 0, "mixer", "rot", "dims"), 7), (("layers", 0, "mixer", "rot", "base"), 1.0), (("layers", 2, "mixer", "mask", "size"), 0),
    (("layers", 0, "mlp", "kind"), "mix"), (("layers", 0, "mlp", "router", "top"), 5), (("layers", 0, "mlp", "router", "groups", "count"), 3),
    (("layers", 0, "mlp", "router", "groups", "keep"), 5), (("layers", 1, "mlp", "ff"), 0), (("layers", 1, "mixer", "tau"), 0.0),
    (("max_positions",), None), (("norm", "eps"), -1.0), (("residual_mult",), "x"), (("layers",), []),
])
def test_refusals(path, value):
    cfg = copy.deepcopy(sc.S1)
    o = cfg
    for key in path[:-1]:
        o = o[key]
    o[path[-1]] = value
    with pytest.raises(ConfigError):
        ZusotarConfig.from_dict(cfg)


def test_a_schedule_averages_behind_every_entry_up_to_the_last_that_does():
    from dataclasses import replace
    spec = zusotar_model_spec(ZusotarConfig.from_dict(sc.S1))
    spec.validate()
    for change in ({1: None}, {2: "l1.dwa"}, {0: "nothing"}):
        bad = replace(spec, schedule=[replace(e, average=change.get(i, e.average)) for i, e in enumerate(spec.schedule)])
        with pytest.raises(ValueError):
            bad.validate()
    replace(spec, schedule=[replace(e, average=e.average if i < 3 else None) for i, e in enumerate(spec.schedule)]).validate()


def test_norm_weights_stored_around_zero_and_the_factor():
    from coheryn_ai_studio_b200.parts.norm import RMSNorm
    w = torch.tensor([0.5, -0.25, 0.0, 2.0], dtype=torch.bfloat16)
    for offset, factor in ((1.0, 1.0), (1.0, 0.3), (0.0, 0.7)):
        n = RMSNorm(CPU, 4, 1e-6, tensor="", offset=offset, factor=factor)
        n.bind({"": w})
        assert n.weight.dtype == torch.float32 and torch.allclose(n.weight, (w.float() + offset) * factor, rtol=1e-7)
    n = RMSNorm(CPU, 4, 1e-6, tensor="")
    n.bind({"": w})
    assert n.weight is w


def test_neighbouring_pairs_become_halves_when_the_weights_are_bound():
    """Rotating the permuted projections in halves gives the same products of queries and keys as rotating the stored ones in
    neighbouring pairs; channels behind the rotated ones keep their place."""
    from coheryn_ai_studio_b200.config.spec import PartSpec
    from coheryn_ai_studio_b200.parts.attention import Attention, LatentAttention, PooledWindowAttention
    from coheryn_ai_studio_b200.parts.base import POSITIONS, build_part
    rng = np.random.default_rng(1)
    width, H, dim, rd, dv, rank, dims = 20, 3, 4, 10, 5, 7, 6
    pos = build_part(POSITIONS, "position", PartSpec("rope_computed", dict(rotary_dim=dims, theta=30.0, pairs="neighbours")), CPU)
    part = LatentAttention(CPU, width, H, dim, rd, dv, rank, 0.3, 1e-6, position=pos)
    W = {n: torch.tensor(rng.normal(0, 1, s.shape)) for n, s in part.tensor_specs().items()}
    part.bind(W)
    h = torch.tensor(rng.normal(0, 1, (9, width)))

    def halves(v):
        f = 30.0 ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
        a = (torch.arange(9, dtype=torch.float64)[:, None] * f).reshape((9,) + (1,) * (v.dim() - 2) + (dims // 2,))
        x, y = v[..., :dims // 2], v[..., dims // 2:dims]
        return torch.cat([x * a.cos() - y * a.sin(), y * a.cos() + x * a.sin(), v[..., dims:]], dim=-1)

    proj = h @ part.w_in.T
    q = proj[:, :H * (dim + rd)].view(9, H, dim + rd)
    d = proj[:, part.kv_col:part.kv_col + rank + rd]
    got = torch.einsum("ihc,jc->hij", halves(q[..., dim:]), halves(d[:, rank:]))
    q0, d0 = (h @ W["q"].T).view(9, H, dim + rd), h @ W["dkv"].T
    want = np.einsum("ihc,jc->hij", plain.rotate_neighbours(q0[..., dim:].numpy(), range(9), dims, 30.0),
                     plain.rotate_neighbours(d0[:, rank:].numpy(), range(9), dims, 30.0))
    assert np.allclose(got.numpy(), want, atol=1e-9) and torch.allclose(q[..., :dim], q0[..., :dim])
    assert torch.allclose(d[:, :rank], d0[:, :rank]) and torch.allclose(d[:, rank + dims:], d0[:, rank + dims:])
    for build in (lambda: PooledWindowAttention(CPU, 8, 1, 1, 8, 8, 1.0, position=pos),
                  lambda: Attention(CPU, 8, 1, 1, 8, False, False, None, 1.0, position=pos)):
        with pytest.raises(ValueError):
            build()


def test_options_that_do_not_go_together_are_refused():
    from coheryn_ai_studio_b200.parts.attention import PooledWindowAttention
    from coheryn_ai_studio_b200.parts.recurrent import GatedLinearAttention
    from coheryn_ai_studio_b200.parts.routed import RoutedExperts
    with pytest.raises(ValueError):
        PooledWindowAttention(CPU, 8, 1, 1, 8, 8, 1.0, window=4, pool=2, log_bias=True)
    with pytest.raises(ValueError):
        RoutedExperts(CPU, 8, 8, 4, 2, selection="top_softmax", renormalize=False)
    with pytest.raises(ValueError):
        RoutedExperts(CPU, 8, 8, 4, 2, selection="sigmoid_top", group_score="three")
    with pytest.raises(ValueError):
        GatedLinearAttention(CPU, 8, 1, 8, 8, 0.0, 1e-6)


# ------------------------------------------------------------------------------------------ the plain pieces
def test_plain_depth_average_and_norms():
    X = [np.full((2, 3), v) for v in (1.0, 10.0, 100.0)]
    assert np.allclose(plain.depth_average(X, [0.5, -1.0, 2.0]), 0.5 - 10.0 + 200.0)
    assert np.allclose(plain.rms_around_zero(np.array([[3.0, -3.0]]), np.array([0.0, 1.0]), 0.0), [[1.0, -2.0]])
    assert np.allclose(plain.rms_around_zero(np.array([[0.0, 0.0]]), np.array([0.0, 1.0]), 1e-6), 0.0)


def test_plain_log_bias_window_on_a_hand_made_case():
    """Equal products of queries and keys: the weights are powers of 1 + r2 d inside the window."""
    T, window, r1, r2 = 9, 4, np.array([2.0, 0.0]), np.array([0.5, 3.0])
    q, k, v = np.zeros((T, 2, 1)), np.zeros((T, 1, 1)), np.eye(T).reshape(T, 1, T)
    out = plain.attend_log_bias(q, k, v, window, 1.0, r1, r2)
    for i in range(T):
        seen = [j for j in range(T) if 0 <= i - j < window]
        for h in range(2):
            w = np.zeros(T)
            w[seen] = [(1.0 + r2[h] * (i - j)) ** -r1[h] for j in seen]
            assert np.allclose(out[i, h], w / w.sum()), (i, h)


def test_plain_linear_attention_on_a_hand_made_case():
    """Constant decays, one key channel per value channel: every channel is a geometric sum."""
    T, dk = 7, 3
    a = np.array([0.0, 0.5, 1.0])
    with np.errstate(divide="ignore"):
        la = np.tile(np.log(a), (T, 1))[:, None, :]
    one = np.ones((T, 1, dk))
    out = plain.linear_attention_scan(one, one, np.tile(np.arange(1.0, T + 1)[:, None, None], (1, 1, 2)), la)
    for t in range(T):
        want = sum(sum(a[d] ** (t - s) * (s + 1.0) for s in range(t + 1)) for d in range(dk))
        assert np.allclose(out[t, 0], want), t


def test_plain_router_takes_the_best_groups_by_their_two_largest_scores():
    logit = lambda p: np.log(p / (1 - p))
    # group 0 has the largest score, group 1 the two largest together, group 2 neither
    s = np.array([[0.9, 0.1, 0.1, 0.6, 0.55, 0.2, 0.5, 0.4, 0.3]])
    W = {"r.router": np.eye(9)}
    ids, w = plain.route(logit(s), W, "r.", {"experts": 9, "top": 2, "groups": {"count": 3, "keep": 1}})
    assert ids.tolist() == [[3, 4]] and np.allclose(w, [[0.6, 0.55]])            # the scores as they are
    ids, w = plain.route(logit(s), W, "r.", {"experts": 9, "top": 3, "groups": {"count": 3, "keep": 2}})
    assert ids.tolist() == [[0, 3, 4]] and np.allclose(w, [[0.9, 0.6, 0.55]])
    ids, _ = plain.route(logit(s), W, "r.", {"experts": 9, "top": 2, "groups": {"count": 9, "keep": 3}})    # groups of one
    assert ids.tolist() == [[0, 3]]
    ids, _ = plain.route(logit(s), W, "r.", {"experts": 9, "top": 4})
    assert ids.tolist() == [[0, 3, 4, 6]]


def test_plain_rotation_of_neighbours_keeps_products_of_equal_distance():
    rng = np.random.default_rng(3)
    q, k = np.tile(rng.normal(0, 1, (1, 1, 8)), (40, 1, 1)), np.tile(rng.normal(0, 1, (1, 1, 8)), (40, 1, 1))
    a, b = plain.rotate_neighbours(q, range(40), 6, 20.0), plain.rotate_neighbours(k, range(40), 6, 20.0)
    s = a[:, 0] @ b[:, 0].T
    for d in range(-39, 40):
        diag = np.diagonal(s, d)
        assert np.allclose(diag, diag[0])
    assert np.allclose(a[:, 0, 6:], q[:, 0, 6:]) and np.allclose(a[1, 0, :2], [q[0, 0, 0] * np.cos(1) - q[0, 0, 1] * np.sin(1),
                                                                              q[0, 0, 1] * np.cos(1) + q[0, 0, 0] * np.sin(1)])
