"""The Vilazen configuration on the CPU: what is read, what is refused, the layout as parts, the tensor names, the cache with
kept first positions, what the parts do to their weights, and the plain implementation's own pieces against hand-made cases."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_vilazen as plain
import vilazen_cases as vc
from coheryn_ai_studio_b200.cache import CacheManager
from coheryn_ai_studio_b200.config import ConfigError, architecture_for
from coheryn_ai_studio_b200.config.vilazen import VilazenConfig, vilazen_model_spec
from coheryn_ai_studio_b200.parts.base import FixedState, PagedKV, Runtime
from coheryn_ai_studio_b200.parts.model import DecoderModel

CPU = Runtime(torch.float32, torch.device("cpu"))


def model_of(cfg):
    return DecoderModel(vilazen_model_spec(VilazenConfig.from_dict(cfg)), CPU)


def test_round_trip_and_registry():
    for cfg, _ in vc.CASES.values():
        c = VilazenConfig.from_dict(cfg)
        assert VilazenConfig.from_dict(c.to_dict()) == c
        assert architecture_for(cfg).name == "Vilazen"
        d = architecture_for(cfg).describe(c)
        assert d["capabilities"]["fixed_state_bytes_per_request"] > 0 and d["layers"] == len(cfg["layers"])
    bounded = VilazenConfig.from_dict(dict(vc.V1, max_positions=700))
    assert bounded.max_positions == 700 and VilazenConfig.from_dict(bounded.to_dict()) == bounded


def test_layout_tensor_names_and_cache():
    m = model_of(vc.V1)
    specs = m.tensor_specs()
    assert {"embed", "embed.norm", "head", "final.norm", "l0.norm1", "l0.mix.left.q", "l0.mix.left.q.b", "l0.mix.left.k.b", "l0.mix.left.v.b",
            "l0.mix.left.sink", "l0.mix.left.g", "l0.mix.left.o", "l0.mix.right.q", "l0.mix.right.g", "l0.mix.right.norm", "l0.mix.right.o",
            "l0.mlp.up", "l0.mlp.down", "l1.mix.q.norm", "l1.mix.k.norm", "l1.mix.vmix", "l1.mix.g", "l4.mix.vmix", "l3.mix.dkv", "l3.mix.uk"} <= set(specs)
    assert not {"l0.mix.right.q.b", "l0.mix.left.q.norm", "l1.mix.q.b", "l1.mix.sink", "l2.mix.vmix", "l2.mlp.up", "l3.mix.sink", "l3.mix.g",
                "l0.mlp.gate", "l0.norm2"} & set(specs)
    assert specs["l1.mix.vmix"].shape == () and specs["l1.mix.q.norm"].shape == (4 * 32,) and specs["l1.mix.k.norm"].shape == (2 * 32,)
    assert specs["l1.mix.g"].shape == (4, 64) and specs["l0.mix.right.g"].shape == (3 * 32, 64) and specs["l0.mix.right.norm"].shape == (3 * 32,)
    assert m.cache_requirements() == [
        (PagedKV(2, 32, None, 16), FixedState((3 * 16 * 32,), torch.float32)), PagedKV(2, 32, 24, 16, keep_first=5),
        PagedKV(1, 16, 11, 48, keep_first=16), PagedKV(1, 64, 21, 0), PagedKV(1, 16, 40, 32)]
    assert [l.mixer.value_mix if hasattr(l.mixer, "value_mix") else None for l in m.layers] == [None, "first", None, None, "later"]
    assert all(p.children[0][1].position.rotary_dim == 16 and p.children[1][1].decay == (0.5, 0.97, 1.0) for p in [m.layers[0].mixer])


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "conv"), (("layers", 1, "mixer", "kv_heads"), 3), (("layers", 1, "mixer", "rot", "dims"), 34),
    (("layers", 1, "mixer", "rot", "dims"), 7), (("layers", 1, "mixer", "rot", "base"), 1.0), (("layers", 1, "mixer", "mask", "size"), 0),
    (("layers", 1, "mixer", "mask", "keep_first"), -1), (("layers", 1, "mixer", "v_mix"), 1), (("layers", 4, "mixer", "vdim"), 48),
    (("layers", 0, "mixer", "right", "decay"), [0.5, 0.9]), (("layers", 0, "mixer", "right", "decay"), [0.5, 0.9, 1.1]),
    (("layers", 0, "mixer", "right", "decay"), [0.5, -0.1, 1.0]), (("layers", 0, "mixer", "left_scale"), "x"), (("layers", 0, "mixer", "left", "rot"), None),
    (("layers", 3, "mixer", "rot", "dims"), 18), (("layers", 3, "mixer", "mask", "keep_first"), 2), (("layers", 0, "mlp", "kind"), "moe"),
    (("layers", 0, "mlp", "ff"), 0), (("norm", "eps"), -1.0), (("width",), None), (("layers",), []),
])
def test_refusals(path, value):
    cfg = copy.deepcopy(vc.V1)
    o = cfg
    for key in path[:-1]:
        o = o[key]
    o[path[-1]] = value
    with pytest.raises(ConfigError):
        VilazenConfig.from_dict(cfg)


def test_options_that_do_not_go_together_are_refused():
    from coheryn_ai_studio_b200.parts.attention import LatentAttention, MapsAttention
    from coheryn_ai_studio_b200.parts.feedforward import MLP
    from coheryn_ai_studio_b200.parts.recurrent import LightningAttention
    for build in (lambda: MapsAttention(CPU, 8, 1, 1, 8, 8, 1.0, keep_first=3), lambda: MapsAttention(CPU, 8, 1, 1, 8, 8, 1.0, window=4, chunk=4, keep_first=3),
                  lambda: MapsAttention(CPU, 8, 1, 1, 8, 8, 1.0, own_kv=False, value_mix="later"), lambda: MapsAttention(CPU, 8, 1, 1, 8, 8, 1.0, value_mix="all"),
                  lambda: MapsAttention(CPU, 8, 1, 1, 8, 8, 1.0, qk_norm="tail"), lambda: LatentAttention(CPU, 8, 1, 8, 2, 8, 8, 1.0, 1e-6, window=0),
                  lambda: LightningAttention(CPU, 8, 2, 8, 8, (0.5,), 1e-6), lambda: LightningAttention(CPU, 8, 1, 8, 8, (1.5,), 1e-6),
                  lambda: CacheManager([PagedKV(1, 4, None, keep_first=2)], [None], torch.float32, "cpu", num_pages=4)):
        with pytest.raises(ValueError):
            build()
    from coheryn_ai_studio_b200.ops import KernelError
    with pytest.raises(KernelError):
        MLP(CPU, 8, 8, "relu")


def test_neighbouring_pairs_become_halves_when_the_weights_are_bound():
    """Rotating the permuted projections in halves gives the same products of queries and keys as rotating the stored ones in
    neighbouring pairs: rows, biases and norm weights move together, per head; values and gates keep their place."""
    from coheryn_ai_studio_b200.config.spec import PartSpec
    from coheryn_ai_studio_b200.parts.attention import MapsAttention
    from coheryn_ai_studio_b200.parts.base import POSITIONS, build_part
    rng = np.random.default_rng(1)
    width, H, G, dk, dv, dims = 14, 4, 2, 9, 5, 6
    pos = build_part(POSITIONS, "position", PartSpec("rope_computed", dict(rotary_dim=dims, theta=30.0, pairs="neighbours")), CPU)
    part = MapsAttention(CPU, width, H, G, dk, dv, 0.3, qkv_bias=True, qk_norm="projection", gate=True, learned_sink=True, position=pos)
    W = {n: torch.tensor(rng.normal(0, 1, s.shape)) for n, s in part.tensor_specs().items()}
    part.bind(W)
    h = torch.tensor(rng.normal(0, 1, (7, width)))
    proj = h @ part.w_in.T + part.b_in.double()

    def halves(v):
        a = (torch.arange(7, dtype=torch.float64)[:, None] * 30.0 ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)).view(7, 1, -1)
        x, y = v[..., :dims // 2], v[..., dims // 2:dims]
        return torch.cat([x * a.cos() - y * a.sin(), y * a.cos() + x * a.sin(), v[..., dims:]], dim=-1)

    q = halves((proj[:, :H * dk] * part.q_norm).view(7, H, dk))
    k = halves((proj[:, H * dk:(H + G) * dk] * part.k_norm).view(7, G, dk))
    n = {m: W[m].numpy() for m in W}
    q0 = plain.rotate_neighbours(((h.numpy() @ n["q"].T + n["q.b"]) * n["q.norm"]).reshape(7, H, dk), range(7), dims, 30.0)
    k0 = plain.rotate_neighbours(((h.numpy() @ n["k"].T + n["k.b"]) * n["k.norm"]).reshape(7, G, dk), range(7), dims, 30.0)
    assert np.allclose(torch.einsum("ihc,jgc->hgij", q, k).numpy(), np.einsum("ihc,jgc->hgij", q0, k0), atol=1e-6)
    at = (H + G) * dk
    assert np.allclose(proj[:, at:at + G * dv].numpy(), h.numpy() @ n["v"].T + n["v.b"], atol=1e-6)
    assert np.allclose(proj[:, at + G * dv:].numpy(), h.numpy() @ n["g"].T, atol=1e-6)


def test_powers_of_the_decays():
    from coheryn_ai_studio_b200 import ops
    p = ops.decay_powers([0.0, 0.25, 1.0 - 1e-9, 1.0], "cpu")
    assert p.shape == (4, 2, ops.LIGHTNING_CHUNK + 1) and p[:, 0, 0].tolist() == [1.0] * 4 and p[:, 1, 0].tolist() == [0.0] * 4
    assert p[0, 0, 1:].tolist() == [0.0] * ops.LIGHTNING_CHUNK and p[0, 1, 1:].tolist() == [-1.0] * ops.LIGHTNING_CHUNK
    assert p[1, 0, 3].item() == 0.25 ** 3 and p[3, 1].abs().max() == 0.0
    assert math.isclose(p[2, 1, 64].item(), -64e-9, rel_tol=1e-6)         # what a power near 1 would have lost


def test_an_embedding_norm_stored_around_zero():
    m = model_of(vc.V1)
    W = {n: torch.randn(s.shape) for n, s in m.embedder.tensor_specs().items()}
    m.embedder.bind(W)
    assert torch.allclose(m.embedder.norm, W["embed.norm"] + 1.0) and m.embedder.state_requirement() is None


# ------------------------------------------------------------------------------------------ pages of kept first positions
@pytest.mark.parametrize("window,keep,page", [(9, 5, 4), (9, 4, 4), (3, 13, 4), (1, 1, 8), (20, 40, 16), (7, 0, 4)])
def test_pages_of_kept_positions_stay_while_the_window_passes(window, keep, page):
    """After every commit the request holds exactly the pages of what a later position can still see."""
    pages, n = 24, 90
    m = CacheManager([PagedKV(1, 4, window, keep_first=keep), PagedKV(1, 4, None)], [None, None], torch.float32, "cpu", page_size=page,
                     num_pages=pages, max_requests=2, prefix_reuse=False)
    assert m.admit("a") is not None
    at = 0
    for count in ([1] * 30 + [7, 2, 19, 1, 1, 30]):
        assert m.reserve("a", [1] * count)
        m.commit("a")
        at += count
        table = m.block_table("a", 0)
        for b in range(len(table)):
            seen = any(at - j < window or j < keep for j in range(b * page, min((b + 1) * page, at + 1)))      # by position `at` or a later one
            assert (table[b] >= 0) == seen, (at, b, table)
        assert m.available_pages()[0] == pages - sum(p >= 0 for p in table)
        m.check()
    assert at == n and not m.prefix_reuse
    assert m.reserve("a", [1] * 3)
    m.rollback("a")
    m.check()
    m.free("a")
    m.check()
    assert m.available_pages() == [pages, pages]


def test_groups_differ_by_what_they_keep():
    m = CacheManager([PagedKV(1, 4, 8, keep_first=2), PagedKV(1, 4, 8), PagedKV(1, 4, 8, keep_first=2)], [None] * 3, torch.float32, "cpu",
                     page_size=4, num_pages=8, max_requests=2, prefix_reuse=False)
    assert [g.entries for g in m.groups] == [[0, 2], [1]]


# ------------------------------------------------------------------------------------------ the plain pieces
def test_plain_visible_positions():
    assert plain.visible(6).tolist() == list(range(7))
    assert plain.visible(9, 3).tolist() == [7, 8, 9] and plain.visible(9, 3, 2).tolist() == [0, 1, 7, 8, 9]
    assert plain.visible(9, 3, 8).tolist() == list(range(10)) and plain.visible(1, 1, 5).tolist() == [0, 1] and plain.visible(0, 1, 5).tolist() == [0]


def test_plain_attention_on_a_hand_made_case():
    """Equal scores: the weights count what is visible, and the sink once."""
    T = 8
    q, k, v = np.zeros((T, 2, 1)), np.zeros((T, 1, 1)), np.eye(T).reshape(T, 1, T)
    out = plain.attend(q, k, v, 1.0, size=3, keep_first=2, sinks=np.array([0.0, math.log(4.0)]))
    for i in range(T):
        see = sorted({0, 1, i, i - 1, i - 2} & set(range(i + 1)))
        for h, extra in ((0, 1), (1, 4)):
            want = np.zeros(T)
            want[see] = 1.0 / (len(see) + extra)
            assert np.allclose(out[i, h], want), (i, h)
    assert np.allclose(plain.gate_heads(np.ones((1, 2, 3)), np.array([[0.0, math.log(3.0)]])), [[[0.5] * 3, [0.75] * 3]])


def test_plain_decay_scan_and_value_mixing():
    T = 6
    one = np.ones((T, 2, 1))
    out = plain.decay_scan(one, one, np.arange(1.0, T + 1).reshape(T, 1, 1) * np.ones((1, 2, 1)), [0.0, 0.5])
    for t in range(T):
        assert np.isclose(out[t, 0, 0], t + 1.0) and np.isclose(out[t, 1, 0], sum(0.5 ** (t - s) * (s + 1.0) for s in range(t + 1)))
    assert np.allclose(plain.mix_values(np.array([1.0]), np.array([3.0]), 0.25), 1.5)
    assert np.allclose(plain.gelu(np.array([0.0, 1.0, -1.0])), [0.0, 0.8413447460685429, -0.15865525393145707])


def test_plain_forward_is_causal_and_mixes_the_first_layers_values():
    cfg = vc.V2
    rng = np.random.default_rng(5)
    W = {n: rng.normal(0, 0.3, s.shape) for n, s in model_of(cfg).tensor_specs().items()}
    toks = vc.prompt(3, 20, cfg["vocab"])
    whole = plain.forward(toks, W, cfg)
    assert np.allclose(plain.forward(toks[:11], W, cfg), whole[:11])
    assert np.array_equal(plain.forward(toks, dict(W, **{"l0.mix.vmix": np.array(9.0)}), cfg), whole)        # the first layer's is unused
    assert not np.allclose(plain.forward(toks, dict(W, **{"l2.mix.vmix": np.array(0.9)}), cfg), whole)
