"""The Vilazen decoder on the GPU against the plain implementation (``plain_vilazen.py``): each mechanism's kernels alone,
then whole models through the step function, the cache and the scheduler, in float32 and in bfloat16."""
import types

import numpy as np
import pytest
import torch

import plain_vilazen as plain
import vilazen_cases as vc

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
NAMES = ["V1", "V2", "V3"]
DEV = "cuda:0"
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("vilazen")
    return {n: vc.make_folder(base, n) for n in NAMES}


@pytest.fixture(scope="module")
def models(folders):
    from coheryn_ai_studio_b200.engine import load_model
    cache = {}

    def get(name, dtype):
        if (name, dtype) not in cache:
            cache[(name, dtype)] = load_model(folders[name], dtype)[1]
        return cache[(name, dtype)]
    return get


def vocab(name):
    return vc.CASES[name][0]["vocab"]


def prompt(name, seed, n):
    return vc.prompt(seed, n, vocab(name))


def dev(a, dtype=torch.float32):
    return torch.as_tensor(np.asarray(a), dtype=dtype).to(DEV)


def bf(a):
    return plain.round_bf16(np.asarray(a, dtype=np.float64))


def f32(a):
    return np.asarray(a, dtype=np.float32).astype(np.float64)


def stored(dtype):
    """How test values are rounded so that the device holds them exactly."""
    return bf if dtype == "bfloat16" else f32


def same(a):
    return a


def host(t):
    return t.float().cpu().numpy().astype(np.float64)


def runtime(dtype):
    from coheryn_ai_studio_b200.parts.base import Runtime
    return Runtime(TORCH[dtype], torch.device(DEV))


def bind(part, W, prefix, dtype):
    """Hand a part its tensors from a dict of float64 arrays, kept as the loader keeps them."""
    from coheryn_ai_studio_b200.weights.loader import kept_dtype
    part.bind({n: dev(W[prefix + n]).to(kept_dtype(s, TORCH[dtype], TORCH[dtype])).contiguous() for n, s in part.tensor_specs().items()})
    return part


def rotation(dims, base, dtype="float32"):
    from coheryn_ai_studio_b200.config.spec import PartSpec
    from coheryn_ai_studio_b200.parts.base import POSITIONS, build_part
    return build_part(POSITIONS, "position", PartSpec("rope_computed", dict(rotary_dim=dims, theta=base, pairs="neighbours")), runtime(dtype))


class Pages:
    """A hand-made cache for one attention: requests whose pages are handed out in a scrambled order and full of noise, and
    steps over any runs of their positions.  With a ``window`` the pages that lie wholly between the first ``keep`` positions
    and every window of a step are -1 in its block table, as a cache that has given them back leaves it."""

    def __init__(self, lengths, G, dk, dv, page, dtype, window=None, keep=0, seed=0):
        from coheryn_ai_studio_b200.parts.base import LayerCache
        self.page, self.window, self.keep = page, window, keep
        pages = [-(-n // page) for n in lengths]
        order = np.random.default_rng(seed).permutation(sum(pages) + 3)
        self.table = np.full((len(lengths), max(pages) + 1), -1, dtype=np.int32)
        at = 0
        for r, n in enumerate(pages):
            self.table[r, :n] = order[at:at + n]
            at += n
        noise = lambda *shape: torch.randn(shape, device=DEV).mul_(7.0).to(TORCH[dtype])
        self.k = noise(sum(pages) + 3, G, page, dk)
        self.v = noise(sum(pages) + 3, G, page, dv) if dv else None
        self.cache = LayerCache(kind="paged", group=0, page_size=page, k=self.k, v=self.v, writes=True)

    def step(self, runs):
        """``runs``: (request, first position, tokens) in batch order; the requests' lengths are first + tokens."""
        req = np.concatenate([np.full(n, i) for i, (_, _, n) in enumerate(runs)]).astype(np.int32)
        pos = np.concatenate([np.arange(s, s + n) for _, s, n in runs]).astype(np.int32)
        cu = np.concatenate([[0], np.cumsum([n for _, _, n in runs])]).astype(np.int32)
        tab = np.stack([self.table[r] for r, _, _ in runs])
        if self.window is not None:
            for b, (_, s, _) in enumerate(runs):
                tab[b, -(-self.keep // self.page):max(0, s - self.window + 1) // self.page] = -1
        slots = np.concatenate([self.table[r][np.arange(s, s + n) // self.page] * self.page + np.arange(s, s + n) % self.page
                                for r, s, n in runs]).astype(np.int32)
        kv = [s + n for _, s, n in runs]
        return types.SimpleNamespace(
            num_requests=len(runs), num_tokens=int(cu[-1]), token_req=dev(req, torch.int32), positions=dev(pos, torch.int32),
            cu_q=dev(cu, torch.int32), kv_lens=dev(kv, torch.int32), block_tables=[dev(tab, torch.int32)],
            slots=[dev(slots, torch.int32)], q_lens=[n for _, _, n in runs], kv_lens_host=kv, shared={},
            max_q_len=max(n for _, _, n in runs), max_kv_len=max(kv), prior_positions_settled=True, tail=None, tail_rows=None)


def state_step(runs, slots):
    """A step without pages: ``runs`` as above; ``slots``: the state slot of every request."""
    cu = np.concatenate([[0], np.cumsum([n for _, _, n in runs])]).astype(np.int32)
    return types.SimpleNamespace(num_requests=len(runs), num_tokens=int(cu[-1]), cu_q=dev(cu, torch.int32), shared={},
                                 state_slots=dev([slots[r] for r, _, _ in runs], torch.int32), tail=None, tail_rows=None,
                                 max_q_len=max(n for _, _, n in runs))


def cuts(lengths, portions):
    """Steps of a schedule: request r joins at step r and advances by portions[r][k] tokens in its k-th step."""
    at = [0] * len(lengths)
    steps, k = [], 0
    while any(a < n for a, n in zip(at, lengths)):
        runs = []
        for r, n in enumerate(lengths):
            if at[r] < n and k >= r:
                take = min(portions[r][(k - r) % len(portions[r])], n - at[r])
                runs.append((r, at[r], take))
                at[r] += take
        steps.append(runs)
        k += 1
    return steps


def run_mixer(mixer, hs, steps, make_step, cache, dtype, width, before=None):
    got = [np.zeros((len(h), width)) for h in hs]
    for runs in steps:
        st = make_step(runs)
        if before is not None:
            before(runs, st)
        x = dev(np.concatenate([hs[r][s:s + n] for r, s, n in runs]), TORCH[dtype])
        out = host(mixer.forward(x, st, cache))
        o = 0
        for r, s, n in runs:
            got[r][s:s + n] = out[o:o + n]
            o += n
    return got


def each_kernel(dtype):
    """The attention's kernels in turn: the tcgen05 one for portions with the tensor-core decode kernel, the one over score
    maps for portions, and the float32-arithmetic one."""
    from coheryn_ai_studio_b200 import ops
    for options, maps in ((True, True), (False, True), (True, False)) if dtype == "bfloat16" else ((True, True),):
        ops.set_attention_options(options)
        ops.set_maps_tc(maps)
        try:
            yield f"options {options}, maps {maps}"
        finally:
            ops.set_attention_options(True)
            ops.set_maps_tc(True)


# ------------------------------------------------------------------------------ embedding, feed-forward
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [64, 100, 1100])
def test_embedding_rows_pass_the_norm(dtype, H):
    from coheryn_ai_studio_b200.parts.embedding import PairHashEmbedding
    rng, V, T = np.random.default_rng(H), 50, 33
    W = {"embed": bf(rng.normal(0, 0.02, (V, H))), "embed.norm": bf(rng.normal(0, 0.3, H))}       # small rows: the eps counts
    part = bind(PairHashEmbedding(runtime(dtype), V, H, "embed", norm="embed.norm", norm_offset=1.0, eps=1e-3, compute_copy=False), W, "", dtype)
    ids = rng.integers(0, V, T)
    st = state_step([(0, 0, T)], [0])
    st.token_ids, st.positions, st.token_req = dev(ids, torch.int32), dev(np.arange(T), torch.int32), dev(np.zeros(T), torch.int32)
    out, status = torch.empty((T, H), device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    assert part.forward(st, None, out, status) is None
    want = plain.rms_around_zero(W["embed"][ids], W["embed.norm"], 1e-3)
    assert np.abs(host(out) - want).max() < 2e-5 * np.abs(want).max() and status.item() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff", [(64, 96), (100, 50), (192, 1000), (1024, 2048)])
def test_feed_forward_without_a_gate(dtype, width, ff):
    """Every product kernel with the activation in its epilogue: few rows and many, outputs that are columns of a wider
    buffer, features that no tile divides."""
    from coheryn_ai_studio_b200 import ops
    from coheryn_ai_studio_b200.parts.feedforward import MLP
    rng, r8 = np.random.default_rng(width), stored(dtype)
    W = {"f.up": r8(rng.normal(0, 2.0 / width ** 0.5, (ff, width))), "f.down": r8(rng.normal(0, 1.0 / ff ** 0.5, (width, ff)))}
    part = bind(MLP(runtime(dtype), width, ff, "gelu", tensors=("up", "down"), float32_output=True), W, "f.", dtype)
    tol = 2e-5 if dtype == "float32" else 2e-2
    for T in (1, 5, 24, 50, 100, 300):
        h = r8(rng.normal(0, 1.0, (T, width)))
        act = plain.gelu(h @ W["f.up"].T)
        wide = torch.full((T, ff + 24), 7.0, dtype=TORCH[dtype], device=DEV)
        part.forward_open(dev(h, TORCH[dtype]), None, None, [wide[:, 8:8 + ff]])
        assert np.abs(host(wide[:, 8:8 + ff]) - act).max() <= tol * np.abs(act).max(), T
        assert (wide[:, :8] == 7.0).all() and (wide[:, 8 + ff:] == 7.0).all()
        want = plain.dense(h, W, "f.", r8 if dtype == "bfloat16" else same)
        assert np.abs(host(part.forward(dev(h, TORCH[dtype]), None)) - want).max() <= tol * np.abs(want).max(), T
    if dtype == "bfloat16":
        x, w = dev(rng.normal(0, 1, (300, width)), torch.bfloat16), dev(W["f.up"], torch.bfloat16)
        bias = rng.normal(0, 1, ff)
        pre = host(x) @ W["f.up"].T + f32(bias)
        for fn, rows in ((ops.gemm_bf16_small, 40), (ops.gemm_bf16_tc, 300), (ops.gemm_bf16_tc_pair, 300), (ops.gemm_bf16_tc_few, 12)):
            if width % 8 or (fn is ops.gemm_bf16_tc_pair and ff % 8):
                continue
            for out_dtype in (torch.bfloat16, torch.float32):
                out = torch.empty((rows, ff), dtype=out_dtype, device=DEV)
                fn(x[:rows], w, dev(bias), out, epilogue=16)
                want = plain.gelu(pre[:rows])
                assert np.abs(host(out) - want).max() <= (1e-2 if out_dtype == torch.bfloat16 else 1e-5) * np.abs(want).max(), (fn.__name__, rows, out_dtype)
        ops.check_tc_status(torch.device(DEV))


# ------------------------------------------------------------------------------ norm over a projection, rotation, value mixing
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,dims", [(4, 2, 32, 16, 32), (3, 3, 20, 14, 6), (18, 1, 16, 16, 16), (40, 8, 64, 10, 20), (1, 1, 8, 130, 2)])
def test_projection_norm_rotation_and_mixed_values(dtype, H, G, dk, dv, dims):
    """q and k normalised over ALL their heads at once, rotated at positions up to a million, k and the mixed v written to
    their pages; a row whose one head is loud changes the other heads' rows (one norm for all)."""
    from coheryn_ai_studio_b200 import ops
    rng = np.random.default_rng(H * dk)
    T, page, first = 21, 8, 1_000_003
    pos = rotation(dims, 5000.0)
    order = pos.halves_order() + list(range(dims, dk))
    for start in (0, first):
        pages = Pages([30], G, dk, dv, page, dtype)
        st = pages.step([(0, 0, T)])
        st.positions = dev(np.arange(start, start + T), torch.int32)
        wide = rng.normal(0, 1, (T, (H + G) * dk + G * dv + 3)).astype(np.float32)
        wide[2, :dk] *= 30.0
        wide[3] *= 1e-3                     # the eps inside the root counts
        vf = rng.normal(0, 1, (T, G * dv + 5)).astype(np.float32)
        wq, wk = f32(rng.normal(1, 0.2, H * dk)), f32(rng.normal(1, 0.2, G * dk))
        p, f = dev(wide), dev(vf)
        nq, nk = H * dk, G * dk
        for mix in (None, 0.3, -1.5):
            q = ops.unit_norm_rope_kv_write(p[:, :nq], p[:, nq:nq + nk], p[:, nq + nk:nq + nk + G * dv], dev(wq), dev(wk), 1e-5, st.positions,
                                            pos.frequency_pairs(), dims, 1.0, st.slots[0], pages.k, pages.v, H, G, G, dk, dv, page, TORCH[dtype],
                                            whole_norm=True, v_first=f[:, 2:2 + G * dv] if mix is not None else None, mix=mix or 0.0)
            def turned(z, w, n):            # the kernel turns halves: neighbours of the channels in the other order
                z = plain.rms(z.astype(np.float64), 1e-5) * w
                back = np.zeros((T, n, dk))
                back[..., order] = z.reshape(T, n, dk)
                return plain.rotate_neighbours(back, np.arange(start, start + T), dims, 5000.0)[..., order]
            want_q, want_k = turned(wide[:, :nq], wq, H), turned(wide[:, nq:nq + nk], wk, G)
            v = wide[:, nq + nk:nq + nk + G * dv].astype(np.float64)
            want_v = v if mix is None else plain.mix_values(v, vf[:, 2:2 + G * dv].astype(np.float64), mix)
            tol = 1e-5 if dtype == "float32" else 8e-3
            assert np.abs(host(q).reshape(T, H, dk) - want_q).max() <= tol * np.abs(want_q).max()
            for t in range(T):
                page_no, off = pages.table[0][t // page], t % page
                assert np.abs(host(pages.k[page_no, :, off]) - want_k[t]).max() <= tol * np.abs(want_k).max(), t
                assert np.abs(host(pages.v[page_no, :, off]) - want_v[t].reshape(G, dv)).max() <= tol * np.abs(want_v).max(), t


# ------------------------------------------------------------------------------ attention: windows that keep the first positions
def run_attention(q, k, v, lengths, steps, page, scale, dtype, G, size=None, keep=0, sinks=None, gates=None, factor=1.0):
    """Write k and v as they are, attend; rows [length][H, dv] per request."""
    from coheryn_ai_studio_b200 import ops
    H, dk, dv = q[0].shape[1], q[0].shape[2], v[0].shape[2]
    pages = Pages(lengths, G, dk, dv, page, dtype, window=size, keep=keep, seed=len(steps))
    got = [np.zeros((n, H, dv)) for n in lengths]
    for runs in steps:
        st = pages.step(runs)
        rows = [np.concatenate([a[r][s:s + n].reshape(n, -1) for r, s, n in runs]) for a in (q, k, v)]
        qd, kd, vd = (p for p in dev(np.concatenate(rows, axis=1)).split([r.shape[1] for r in rows], dim=1))
        qq = ops.unit_norm_rope_kv_write(qd, kd, vd, None, None, 1e-6, st.positions, None, 0, 1.0, st.slots[0], pages.k, pages.v, H, G, G,
                                         dk, dv, page, TORCH[dtype])
        out = torch.full((qq.shape[0], H * dv + 8), 3.0, dtype=TORCH[dtype], device=DEV)
        g = dev(np.concatenate([gates[r][s:s + n] for r, s, n in runs])) if gates is not None else None
        ops.attention_maps(qq, out[:, 4:4 + H * dv], pages.k, pages.v, st, 0, H, G, dk, dv, 1, page, size, None, sinks is not None, scale, 0.0,
                           False, 1e-6, factor, sink_scores=dev(sinks) if sinks is not None else None, head_gates=g, keep_first=keep)
        assert (out[:, :4] == 3.0).all() and (out[:, 4 + H * dv:] == 3.0).all()
        o = 0
        for r, s, n in runs:
            got[r][s:s + n] = host(out[o:o + n, 4:4 + H * dv]).reshape(n, H, dv)
            o += n
    ops.check_tc_status(torch.device(DEV))
    return got


WINDOWS = [(24, 5, 16, 4, 2, 32, 16), (7, 3, 16, 3, 3, 20, 14), (5, 8, 8, 6, 2, 16, 48), (1, 1, 16, 6, 1, 16, 48), (36, 64, 64, 2, 1, 80, 96),
           (72, 37, 16, 8, 4, 48, 48), (33, 32, 8, 4, 1, 64, 128), (6, 41, 16, 18, 1, 16, 16), (40, 0, 16, 4, 2, 96, 64), (130, 6, 32, 5, 1, 128, 128),
           (3, 150, 16, 2, 2, 144, 160), (9, 129, 128, 4, 4, 16, 16)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep,page,H,G,dk,dv", WINDOWS)
def test_one_key_that_stands_out_at_the_windows_edges(dtype, size, keep, page, H, G, dk, dv):
    """A marked position j*: its key and the queries of ALL rows carry one large component, so a row puts nearly all its
    weight on j* while it sees it and none once it does not.  Marks at position 0, the last kept position, the first that is
    not kept, on both sides of page borders and far in; whole, in portions and decoded, over block tables whose passed pages
    are gone."""
    T = 290
    rng, r8 = np.random.default_rng(size * 100 + dk), stored(dtype)
    base = [r8(rng.normal(0, 0.3, (T, n, d))) for n, d in ((H, dk), (G, dk))]
    v = r8(rng.normal(0, 1.0, (T, G, dv)))
    schedules = ([[(0, 0, T)]], cuts([T], [[40, 1, 1, 1, 17, 2, 1, 3, 64, 1, 1, 1, 1, 6, 90]]), [[(0, t, 1)] for t in range(T)])
    tol = 2e-5 if dtype == "float32" else 3e-2
    for marks in ([0, 160], [max(keep - 1, 0)], [keep, 128]):
        q, k = base[0].copy(), base[1].copy()
        q[:, :, 0] = 9.0
        for j in marks:
            k[j, :, 0] = 9.0
        want = plain.attend(q, k, v, 0.3, size, keep)
        for j in marks:          # the first row that does not see the mark any more differs from the one before
            if j >= keep and j + size < T and not any(m != j and (m < keep or m > j) for m in marks):
                assert np.abs(want[j + size - 1] - want[j + size]).max() > 0.2, j
        for label in each_kernel(dtype):
            for steps in schedules:
                got = run_attention([q], [k], [v], [T], steps, page, 0.3, dtype, G, size, keep)[0]
                d = np.abs(got - want).max(axis=(1, 2))
                assert d.max() <= tol * np.abs(want).max(), (label, marks, len(steps), int(d.argmax()), d.max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,page,size,keep", [(4, 2, 32, 16, 16, None, 0), (6, 2, 10, 22, 8, None, 0), (2, 2, 64, 48, 64, 50, 9), (5, 1, 128, 128, 16, None, 0),
                                                      (6, 2, 96, 64, 16, 100, 70)])
def test_sinks_gates_and_a_factor_with_far_keys(dtype, H, G, dk, dv, page, size, keep):
    """Sinks from far below to far above the scores, gates per head from shut to open, a factor on the output; requests of
    unequal lengths, portions beside single tokens; a far key that the last rows single out among hundreds."""
    rng, r8 = np.random.default_rng(dk + dv), stored(dtype)
    lengths = [311, 45, 130]
    q = [r8(rng.normal(0, 1.0, (n, H, dk))) for n in lengths]
    k = [r8(rng.normal(0, 1.0, (n, G, dk))) for n in lengths]
    v = [r8(rng.normal(0, 1.0, (n, G, dv))) for n in lengths]
    k[0][3, :, 1] = 12.0
    q[0][-60:, :, 1] = 12.0
    sinks, gates = f32(np.linspace(-9.0, 25.0, H)), [f32(rng.normal(0, 4.0, (n, H))) for n in lengths]
    scale = 0.5 / dk ** 0.5
    want = [plain.gate_heads(plain.attend(a, b, c, scale, size, keep, sinks), g) * 0.6 for a, b, c, g in zip(q, k, v, gates)]
    alone = plain.attend(q[0], np.concatenate([k[0][:3], 0 * k[0][3:4], k[0][4:]]), v[0], scale, size, keep, sinks)
    if size is None or keep > 3:
        assert np.abs(plain.gate_heads(alone, gates[0])[-60:] * 0.6 - want[0][-60:]).max() > 0.2            # the far key shows
    for label in each_kernel(dtype):
        for steps in (cuts(lengths, [[33, 2, 1, 217, 1, 1, 1, 40, 2, 1, 1, 1], [5, 1, 1, 20, 1], [1, 1, 128]]), cuts(lengths, [[311], [45], [130]])):
            got = run_attention(q, k, v, lengths, steps, page, scale, dtype, G, size, keep, sinks, gates, 0.6)
            for g, w in zip(got, want):
                for h in range(H):      # head by head: a head whose sink takes nearly all is small
                    d = np.abs(g[:, h] - w[:, h]).max()
                    assert d <= (3e-5 if dtype == "float32" else 2e-2) * max(np.abs(w[:, h]).max(), 1e-3), (label, h, d)


def test_portions_split_over_clusters_and_paired_row_tiles_give_the_same_rows():
    """The tcgen05 kernel's ways to share a row tile's keys over CTAs, and two row tiles per CTA, with kept positions."""
    from coheryn_ai_studio_b200 import ops
    rng = np.random.default_rng(3)
    H, G, dk, dv, page, T, size, keep = 4, 2, 64, 96, 16, 700, 300, 140
    q, k, v = bf(rng.normal(0, 1, (T, H, dk))), bf(rng.normal(0, 1, (T, G, dk))), bf(rng.normal(0, 1, (T, G, dv)))
    q[:, :, 0] = 6.0
    for j in (0, 139, 140, 400):
        k[j, :, 0] = 6.0
    sinks = f32(rng.normal(0, 1, H))
    lib = ops.attention_options_lib(dk, dv)
    for window, kept in ((None, 0), (size, keep)):
        want = plain.attend(q, k, v, 0.2, window, kept, sinks)
        try:
            for cluster, two in ((1, 0), (2, 0), (4, 0), (8, 0), (1, 1)):
                lib.coheryn_attention_options_set_cluster(cluster)
                lib.coheryn_attention_options_set_two_tiles(two)
                for steps in ([[(0, 0, T)]], [[(0, 0, 450)], [(0, 450, 250)]]):
                    got = run_attention([q], [k], [v], [T], steps, page, 0.2, "bfloat16", G, window, kept, sinks)[0]
                    d = np.abs(got - want).max(axis=(1, 2))
                    assert d.max() <= 2e-2 * np.abs(want).max(), (window, cluster, two, len(steps), int(d.argmax()), d.max())
        finally:
            lib.coheryn_attention_options_set_cluster(0)
            lib.coheryn_attention_options_set_two_tiles(2)


MIXERS = [({"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 16, "mask": {"size": 24, "keep_first": 5}, "scale": 0.3, "rot": {"dims": 32, "base": 500.0}}, 64, 16),
          ({"heads": 3, "kv_heads": 3, "dim": 20, "vdim": 14, "mask": {"size": 7, "keep_first": 3}, "scale": 0.4, "rot": {"dims": 6, "base": 77.0}}, 100, 16),
          ({"heads": 18, "kv_heads": 1, "dim": 16, "vdim": 16, "mask": {"size": 6, "keep_first": 37}, "scale": 0.3, "rot": {"dims": 16, "base": 50.0}}, 64, 8),
          ({"heads": 2, "kv_heads": 1, "dim": 144, "vdim": 112, "mask": {"size": 50}, "scale": 0.1, "rot": {"dims": 144, "base": 1e6}}, 128, 64)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,width,page", MIXERS)
def test_window_attention_mixer_mixes_an_earlier_layers_values(dtype, m, width, page):
    """The whole mixer for two requests cut into portions, as the first layer that mixes and as a later one."""
    from coheryn_ai_studio_b200.parts.attention import MapsAttention
    rng, r8 = np.random.default_rng(m["dim"] + m["vdim"]), stored(dtype)
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    W = {n: r8(w) for n, w in {
        "m.q": rng.normal(0, 0.25, (H * dk, width)), "m.k": rng.normal(0, 0.25, (G * dk, width)), "m.v": rng.normal(0, 0.25, (G * dv, width)),
        "m.g": rng.normal(0, 0.25, (H, width)), "m.o": rng.normal(0, 0.25, (width, H * dv)), "m.q.norm": rng.normal(1, 0.2, H * dk),
        "m.k.norm": rng.normal(1, 0.2, G * dk), "m.vmix": np.array(0.375)}.items()}
    lengths = [239, 30]
    hs = [r8(rng.normal(0, 1.0, (n, width))) for n in lengths]
    firsts = [f32(rng.normal(0, 1.5, (n, G * dv))) for n in lengths]
    rounder = r8 if dtype == "bfloat16" else same
    steps = cuts(lengths, [[33, 2, 1, 17, 1, 1, 1, 40, 2, 1, 1, 1, 90], [5, 1, 1, 20, 1]])
    for role in ("first", "later"):
        mixer = bind(MapsAttention(runtime(dtype), width, H, G, dk, dv, m["scale"], window=m["mask"]["size"], keep_first=m["mask"].get("keep_first", 0),
                                   qk_norm="projection", gate=True, value_mix=role, eps=1e-6, position=rotation(m["rot"]["dims"], m["rot"]["base"], dtype),
                                   float32_output=True), W, "m.", dtype)
        want = [plain.windowed_attention(h, W, "m.", dict(m, v_mix=True), 1e-6, rounder, {} if role == "first" else {"v": f}) for h, f in zip(hs, firsts)]
        pages = Pages(lengths, G, dk, dv, page, dtype, window=m["mask"]["size"], keep=m["mask"].get("keep_first", 0), seed=width)

        def before(runs, st):
            if role == "later":
                st.shared["v_first"] = dev(np.concatenate([firsts[r][s:s + n] for r, s, n in runs]))

        got = run_mixer(mixer, hs, steps, pages.step, pages.cache, dtype, width, before=before)
        for g, w in zip(got, want):
            tol = 4e-5 if dtype == "float32" else 4e-2
            assert np.abs(g - w).max() <= tol * np.abs(w).max(), (role, np.abs(g - w).max() / np.abs(w).max())
    with pytest.raises(ValueError):
        mixer.forward(dev(hs[1][:2], TORCH[dtype]), pages.step([(1, 0, 2)]), pages.cache)           # nothing to mix with


# ------------------------------------------------------------------------------ linear attention with a constant decay
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,dk,dv,decay", [(64, 16, 32, [0.5, 0.97, 1.0]), (100, 12, 7, [0.0, 0.9]), (48, 48, 144, [0.999]), (64, 130, 20, [0.6, 0.9999]),
                                               (32, 257, 64, [0.95]), (64, 64, 128, [0.2, 0.8, 0.99, 1.0])])
def test_lightning_attention_in_portions_and_decoded(dtype, width, dk, dv, decay):
    """Two requests in portions of many sizes (across chunks of 64, down to one token, beside each other) over state slots
    full of noise.  Decays from 0 (only the token itself) to 1 (a loud first token is there for good)."""
    from coheryn_ai_studio_b200.parts.base import LayerCache
    from coheryn_ai_studio_b200.parts.recurrent import LightningAttention
    rng, r8, H = np.random.default_rng(dk * dv), stored(dtype), len(decay)
    W = {n: r8(rng.normal(0, 0.2, s)) for n, s in {"m.q": (H * dk, width), "m.k": (H * dk, width), "m.v": (H * dv, width), "m.g": (H * dv, width),
                                                   "m.o": (width, H * dv)}.items()}
    W["m.norm"] = r8(rng.normal(1, 0.2, H * dv))
    mixer = bind(LightningAttention(runtime(dtype), width, H, dk, dv, decay, 1e-6, out_scale=0.5), W, "m.", dtype)
    lengths = [331, 45]
    hs = [r8(rng.normal(0, 1.0, (n, width))) for n in lengths]
    hs[0][0] = r8(hs[0][0] * 12.0)
    m = {"heads": H, "dim": dk, "vdim": dv, "decay": decay}
    want = [0.5 * plain.lightning_attention(h, W, "m.", m, 1e-6) for h in hs]
    if max(decay) > 0.99:
        lost = 0.5 * plain.lightning_attention(np.concatenate([hs[0][1:2], hs[0][1:]]), W, "m.", m, 1e-6)
        assert np.abs(lost[-1] - want[0][-1]).max() > 0.003 * np.abs(want[0]).max()             # a lost state would show
    slots = [3, 1]
    schedules = [cuts(lengths, [[130, 2, 1, 67, 31, 33, 1, 1, 1, 64], [7, 1, 2, 30, 1]]), cuts(lengths, [[331], [45]]),
                 cuts(lengths, [[64, 65, 63, 8, 9], [8]])]
    for steps in schedules:
        state = torch.randn((5, H * dk * dv), device=DEV) * 3.0
        fresh = set()

        def admit(runs, st):
            for r, _, _ in runs:
                if r not in fresh:
                    state[slots[r]].zero_()          # what admission does
                    fresh.add(r)

        got = run_mixer(mixer, hs, steps, lambda runs: state_step(runs, slots), LayerCache(kind="state", state=state, writes=True),
                        dtype, width, before=admit)
        for g, w in zip(got, want):
            tol = 4e-5 if dtype == "float32" else 3e-2
            assert np.abs(g - w).max() <= tol * np.abs(w).max(), np.abs(g - w).max() / np.abs(w).max()


def test_linear_attention_long_memories_do_not_drift():
    """A thousand tokens through decays within 1e-4 of 1, one token at a time and in chunks: the error of the state stays at
    float32's rounding, it does not grow with the position."""
    from coheryn_ai_studio_b200 import ops
    rng = np.random.default_rng(4)
    T, H, dk, dv = 1000, 3, 16, 16
    decay = [0.9999, 1.0 - 1e-6, 1.0]
    q, k, v, g = (rng.normal(0, 1, (T, H * d)) for d in (dk, dk, dv, dv))
    o = plain.decay_scan(f32(q).reshape(T, H, dk), f32(k).reshape(T, H, dk), f32(v).reshape(T, H, dv), decay).reshape(T, H * dv)
    want = plain.rms(o, 1e-6) * plain.sigmoid(f32(g))
    powers = ops.decay_powers(decay, DEV)
    for portion in (1, 200, T):
        state = torch.zeros((1, H * dk * dv), device=DEV)
        out = torch.empty((T, H * dv), device=DEV)
        for t in range(0, T, portion):
            s = slice(t, t + portion)
            ops.lightning_attention(dev(q[s]), dev(k[s]), dev(v[s]), dev(g[s]), powers, False, state, state_step([(0, t, portion)], [0]), H, dk, dv,
                                    torch.ones(H * dv, device=DEV), 1e-6, out[s])
        d = np.abs(host(out) - want).max(1)
        assert d.max() <= 3e-5 * np.abs(want).max() and d[-100:].mean() <= 4.0 * d[50:150].mean() + 1e-6, (portion, d.max())


# ------------------------------------------------------------------------------ latent attention over a window
LATENTS = [({"heads": 4, "dim": 32, "rot_dim": 16, "vdim": 16, "kv_rank": 48, "scale": 0.25, "mask": {"size": 21}, "rot": {"dims": 16, "base": 1000.0}}, 64, 16),
           ({"heads": 5, "dim": 12, "rot_dim": 6, "vdim": 10, "kv_rank": 22, "scale": 0.3, "mask": {"size": 1}, "rot": {"dims": 6, "base": 77.0}}, 100, 8),
           ({"heads": 1, "dim": 48, "rot_dim": 64, "vdim": 80, "kv_rank": 272, "scale": 0.1, "mask": {"size": 130}, "rot": {"dims": 64, "base": 5e5}}, 128, 64),
           ({"heads": 18, "dim": 16, "rot_dim": 32, "vdim": 32, "kv_rank": 96, "scale": 0.2, "mask": {"size": 64}, "rot": {"dims": 20, "base": 9.0}}, 64, 16)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,width,page", LATENTS)
def test_latent_attention_mixer_at_its_windows_edges(dtype, m, width, page):
    """The whole mixer for two requests in portions and decoded.  Single tokens share a direction with all queries (in the
    unrotated part), so every row puts most of its weight on one while its window holds it."""
    from coheryn_ai_studio_b200.parts.attention import LatentAttention
    rng, r8 = np.random.default_rng(m["dim"] + m["kv_rank"]), stored(dtype)
    H, dim, rd, vd, rank, size = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["mask"]["size"]
    W = {"m.q": rng.normal(0, 0.03 if rank > 200 else 0.2, (H * (dim + rd), width)), "m.dkv": rng.normal(0, 0.2, (rank + rd, width)), "m.dkv.norm": rng.normal(1, 0.2, rank),
         "m.uk": rng.normal(0, 0.3, (H * dim, rank)), "m.uv": rng.normal(0, 0.3, (H * vd, rank)), "m.o": rng.normal(0, 0.2, (width, H * vd))}
    lengths = [311, 45]
    hs = [rng.normal(0, 1.0, (n, width)) for n in lengths]
    # input 0 makes latent channel 0 and input 1 the queries' component along what latent channel 0 gives every head's keys
    W["m.dkv"][0, 0], W["m.dkv"][rank:, 0], W["m.dkv.norm"][0] = 3.0, 0.0, 1.5
    for h in range(H):
        u = W["m.uk"][h * dim:(h + 1) * dim, 0]
        u[:] = np.sign(u + 1e-9) * 0.5
        W["m.q"][h * (dim + rd):h * (dim + rd) + dim, 1] = u * (8.0 / (m["scale"] * dim))
    hs[0][:, 0], hs[0][:, 1] = 0.0, 1.0
    marks = list(range(2, lengths[0] - size, size + 9))[:5]          # one at a time in any window
    hs[0][marks, 0] = 6.0
    W, hs = {n: r8(w) for n, w in W.items()}, [r8(h) for h in hs]
    rounder = r8 if dtype == "bfloat16" else same
    want = [plain.latent_attention(h, W, "m.", m, 1e-6, rounder) for h in hs]
    wider = plain.latent_attention(hs[0], W, "m.", dict(m, mask={"size": size + 1}), 1e-6, rounder)
    for j in marks:          # a window that is one token off shows at the row behind the edge
        assert np.abs(wider[j + size] - want[0][j + size]).max() > 0.15 * np.abs(want[0]).max(), j
    mixer = bind(LatentAttention(runtime(dtype), width, H, dim, rd, vd, rank, m["scale"], 1e-6, window=size,
                                 position=rotation(m["rot"]["dims"], m["rot"]["base"], dtype)), W, "m.", dtype)
    for label in each_kernel(dtype):
        for steps in (cuts(lengths, [[33, 2, 1, 217, 1, 1, 1, 40, 2, 1, 1, 1], [5, 1, 1, 20, 1]]), cuts(lengths, [[311], [45]]), cuts(lengths, [[1], [1]])):
            pages = Pages(lengths, 1, rank + rd, 0, page, dtype, window=size, seed=width)
            got = run_mixer(mixer, hs, steps, pages.step, pages.cache, dtype, width)
            for g, w in zip(got, want):
                tol = 4e-5 if dtype == "float32" else 5e-2
                assert np.abs(g - w).max() <= tol * np.abs(w).max(), (label, len(steps), np.abs(g - w).max() / np.abs(w).max())


# ------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts(name, dtype, folders, models):
    for i, n in enumerate([1, 2, 23, 97]):
        seq = prompt(name, 30 + i, n)
        r = vc.noisy_replay(folders[name], dtype, 128, models(name, dtype))
        r.step([("r", seq, list(range(n)))], end=["r"])
        vc.check_rows(r.rows, folders[name], {"r": seq}, dtype, f"whole {n}")


def test_layer_outputs_equal_the_plain_layers(folders, models):
    for name in NAMES:
        seq = prompt(name, 3, 29)
        config, w = vc.read_model(folders[name])
        want = []
        plain.forward(seq, w, config, layer_outputs=want)
        r = vc.noisy_replay(folders[name], "float32", 64, models(name, "float32"), layer_outputs=True)
        r.step([("r", seq[:20], [19])])
        r.step([("r", seq[20:], [8])])
        for t in range(29):
            got = r.layers[("r", t)]
            assert len(got) == len(want)
            for i in range(len(want)):
                assert np.abs(got[i] - want[i][t]).max() <= 2e-4 * max(1.0, np.abs(want[i][t]).max()), (name, i, t)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_token_by_token(name, dtype, folders, models):
    n = 120
    seq = prompt(name, 41, n)
    r = vc.noisy_replay(folders[name], dtype, 128, models(name, dtype))
    r.step([("r", seq[:n - 50], list(range(0, n - 50, 3)))])
    for t in range(n - 50, n):
        r.step([("r", [seq[t]], [0])])
    vc.check_rows(r.rows, folders[name], {"r": seq}, dtype, "tail")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_every_token_decoded(name, dtype, folders, models):
    """From the first token on, one by one (the first tokens of a sequence, then a long decode over many pages and windows
    that give their pages back but for the kept ones)."""
    n = 90 if dtype == "bfloat16" else 260
    seq = prompt(name, 42, n)
    r = vc.noisy_replay(folders[name], dtype, 272, models(name, dtype))
    for t in range(n):
        r.step([("r", [seq[t]], [0] if t < 4 or t % 4 == 0 or t > n - 5 else [])])
    vc.check_rows(r.rows, folders[name], {"r": seq}, dtype, "decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_down_to_two_tokens(name, dtype, folders, models):
    portions = [7, 2, 16, 3, 2, 33, 1, 15, 2, 17, 2, 5, 1, 1, 2, 40, 2, 70, 9]
    n = sum(portions)
    seq = prompt(name, 43, n)
    r = vc.noisy_replay(folders[name], dtype, 240, models(name, dtype), page_size=8)
    o = 0
    for p in portions:
        r.step([("r", seq[o:o + p], list(range(p)))])
        o += p
    vc.check_rows(r.rows, folders[name], {"r": seq}, dtype, "portions")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(name, dtype, folders, models):
    """Five requests over three state slots and a pool of 14 pages of 16: portions of some beside single tokens of others;
    a request that ends gives its pages and its slot (with the state it left) to the next, which must not see them."""
    seqs = {f"s{i}": prompt(name, 50 + i, n) for i, n in enumerate([61, 9, 130, 33, 47])}
    r = vc.noisy_replay(folders[name], dtype, 14 * 16, models(name, dtype), max_requests=3)
    at = {k: 0 for k in seqs}

    def take(rid, n):
        toks = seqs[rid][at[rid]:at[rid] + n]
        want = [i for i in range(len(toks)) if (at[rid] + i) % 3 == 0 or at[rid] + i == len(seqs[rid]) - 1]
        at[rid] += len(toks)
        return (rid, toks, want)

    def done(*rids):
        return [x for x in rids if at[x] == len(seqs[x])]

    r.step([take("s0", 20), take("s1", 2)])
    r.step([take("s0", 1), take("s1", 1), take("s2", 50)])
    r.step([take("s0", 40), take("s1", 6), take("s2", 1)], end=["s0", "s1"])
    r.step([take("s2", 1), take("s3", 33)], end=["s3"])
    r.step([take("s4", 2), take("s2", 30)])
    while at["s2"] < 130 or at["s4"] < 47:
        batch = [take(x, 1 if x == "s2" else 5) for x in ("s2", "s4") if at[x] < len(seqs[x])]
        r.step(batch, end=done(*[b[0] for b in batch]))
    assert all(at[k] == len(seqs[k]) for k in seqs)
    vc.check_rows(r.rows, folders[name], seqs, dtype, "mixed")
    assert len(r.cache.requests) == 0 and r.cache.available_pages() == [14] * len(r.cache.groups)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_batched_rows_equal_the_rows_of_each_request_alone(name, dtype, folders, models):
    """What a request's rows are does not depend on what else is in the batch, nor on pages and slots, beyond rounding."""
    a, b = prompt(name, 60, 45), prompt(name, 61, 18)
    alone = vc.noisy_replay(folders[name], dtype, 128, models(name, dtype))
    alone.step([("a", a[:30], list(range(30)))])
    alone.step([("a", a[30:], list(range(15)))])
    both = vc.noisy_replay(folders[name], dtype, 128, models(name, dtype))
    both.step([("b", b[:10], [9]), ("a", a[:30], list(range(30)))])
    both.step([("a", a[30:], list(range(15))), ("b", b[10:], [7])])
    for p in range(45):
        d = np.abs(alone.rows[("a", p)] - both.rows[("a", p)]).max()
        assert d <= (1e-4 if dtype == "float32" else 0.06) * np.std(alone.rows[("a", p)]), (p, d)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_few_wanted_rows_take_the_last_layers_shortcut(name, dtype, folders, models):
    """Steps that want few rows (or none) run the last layer behind its cache or state for those rows only (V1: a window
    attention that mixes values; V3: two mixers side by side; V2's output products do not join, so it has no shortcut): the
    logits equal the plain implementation's, and switching the shortcut off changes nothing beyond rounding."""
    n = 131
    seq, other = prompt(name, 33, n), prompt(name, 34, 40)
    runs = {}
    for shortcut in (True, False):
        r = vc.noisy_replay(folders[name], dtype, 256, models(name, dtype))
        r.runner.tail_shortcut = shortcut
        r.step([("r", seq[:30], [])])
        r.step([("r", seq[30:60], [29, 3]), ("o", other[:20], [19])])
        r.step([("r", seq[60:n - 5], [0]), ("o", other[20:], [])])
        r.step([("r", seq[n - 5:], list(range(5)))])
        assert set(k for k in r.rows if k[0] == "r") == {("r", p) for p in [59, 33, 60] + list(range(n - 5, n))}
        vc.check_rows(r.rows, folders[name], {"r": seq, "o": other}, dtype, f"shortcut {shortcut}")
        runs[shortcut] = r.rows
    assert models(name, dtype).layers[-1].supports_tail == (name != "V2")
    for key, row in runs[True].items():
        assert np.abs(row - runs[False][key]).max() <= (2e-4 * max(1.0, np.std(row)) if dtype == "float32" else 0.08 * np.std(row)), key


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_and_their_expanded_latents(dtype, tmp_path):
    """A prompt of 600 tokens at once (latent rows expanded per head in bfloat16), then portions behind it and decoded tokens,
    through windows longer than a key tile."""
    from coheryn_ai_studio_b200.engine import load_model
    cfg = vc._config(200, 64, 1e-6, [
        vc._latent(2, 16, 16, 16, 112, 150, 300.0, 0.25, 64), vc._both((2, 1, 64, 32, 32, 3000.0, 0.125), (16, 16, [0.9, 0.995]), (0.6, 0.5), None),
        vc._window(2, 1, 32, 16, 200, 9, 16, 5000.0, 0.2, 48), vc._latent(2, 32, 16, 32, 96, None, 10000.0, 0.2, 32),
        vc._window(4, 1, 16, 16, 40, 150, 16, 5000.0, 0.25, None)])
    folder = vc.make_folder(tmp_path, "long", cfg, 71)
    model = load_model(folder, dtype)[1]
    seq = vc.prompt(90, 660, 200)
    r = vc.noisy_replay(folder, dtype, 768, model)
    r.step([("r", seq[:600], list(range(0, 600, 23)) + [599])])
    r.step([("r", seq[600:640], [0, 1, 20, 39])])
    for t in range(640, 660):
        r.step([("r", [seq[t]], [0])])
    vc.check_rows(r.rows, folder, {"r": seq}, dtype, "long")


def test_tensor_core_attention_equals_the_float32_arithmetic_one_in_a_model(folders, models):
    """The same bfloat16 steps with each of the attention's kernels: rows agree within rounding."""
    for name in ("V1", "V3"):
        seq, other = prompt(name, 62, 150), prompt(name, 63, 70)
        rows = {}
        for label in each_kernel("bfloat16"):
            r = vc.noisy_replay(folders[name], "bfloat16", 256, models(name, "bfloat16"))
            r.step([("r", seq[:91], list(range(0, 91, 2)))])
            r.step([("r", seq[91:140], list(range(0, 49, 3))), ("o", other, [69, 5])])
            for t in range(140, 150):
                r.step([("r", [seq[t]], [0])])
            vc.check_rows(r.rows, folders[name], {"r": seq, "o": other}, "bfloat16", label)
            rows[label] = r.rows
        first = next(iter(rows.values()))
        for other_rows in rows.values():
            assert all(np.abs(first[k] - other_rows[k]).max() <= 0.06 * np.std(first[k]) for k in first)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation_through_the_engine(name, dtype, folders):
    """The Python entry point with its scheduler, continuous batching, portions of 16 tokens and decode steps replayed
    from CUDA graphs: every generated token is the plain implementation's first maximum given the tokens before it (in
    bfloat16: or a near tie)."""
    from coheryn_ai_studio_b200.engine import Engine
    eng = Engine.from_folder(folders[name], dtype, context=128, max_num_seqs=3, max_num_batched_tokens=16, page_size=8)
    prompts = [prompt(name, 70 + i, n) for i, n in enumerate((3, 29, 60, 1))]
    res = eng.generate(prompts, max_tokens=16)
    for p, out in zip(prompts, res):
        ids = list(p)
        assert out.completion_tokens == 16 and out.finish_reason == "length"
        for tok in out.token_ids:
            ref = vc.plain_rows(folders[name], ids)[-1]
            best = int(np.argmax(ref))
            if tok != best:
                gap = float(ref[best] - ref[tok]) / float(np.std(ref))
                assert gap <= (1e-3 if dtype == "float32" else 0.15), (name, len(ids), tok, best, gap)
            ids.append(tok)
    eng.cache.check()
    assert len(eng.cache.requests) == 0


def test_trace_program_replays_a_schedule(folders, tmp_path):
    """bin/trace_run on a folder of this design: portions, a second request, an ended request, a step that wants nothing."""
    import json, os, subprocess, sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    name = "V2"
    a, b = prompt(name, 80, 40), prompt(name, 81, 12)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:25], "want": [0, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[25:27], "want": []}, {"id": "b", "tokens": b, "want": [11]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[27:], "want": [12]}], "end": ["a"]}]
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders[name], "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=900)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    V = vocab(name)
    got0 = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, V)
    got1 = np.fromfile(out / "1.f32", dtype="<f4").reshape(1, V)
    got2 = np.fromfile(out / "2.f32", dtype="<f4").reshape(1, V)
    rows = {("a", 0): got0[0], ("a", 24): got0[1], ("b", 11): got1[0], ("a", 39): got2[0]}
    vc.check_rows(rows, folders[name], {"a": a, "b": b}, "float32", "trace")


def test_command_line_runs_and_inspects_the_design(folders):
    import os, subprocess, sys
    from coheryn_ai_studio_b200 import api
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    name = "V1"
    p = prompt(name, 85, 27)
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "coheryn"), "run", folders[name], "--tokens", ",".join(map(str, p)),
                        "--max-tokens", "5", "--context", "64", "--dtype", "float32", "--stream"], capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    got = [int(t) for t in r.stdout.split()]
    ids = list(p)
    for tok in got:
        assert tok == int(np.argmax(vc.plain_rows(folders[name], ids)[-1]))
        ids.append(tok)
    assert api.generate(folders[name], [p], max_tokens=5, context=64, dtype="float32")[0]["token_ids"] == got
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "coheryn"), "models", "inspect", folders[name]], capture_output=True,
                       text=True, timeout=900)
    assert r.returncode == 0 and "Vilazen" in r.stdout, r.stderr[-2000:]


def test_zz_report():
    print(f"\nVilazen rows against the plain implementation: float32 largest |d| = {vc.WORST['float32']:.2e} of the spread; "
          f"bfloat16 largest distance = {vc.WORST['bfloat16']:.2f} of the bound")
