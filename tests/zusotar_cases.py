"""Small Zusotar configurations of the tests (they differ from each other in every size and option), folders of seeded
random weights for them, and the comparison of engine rows with the plain implementation."""
from __future__ import annotations

import json
from typing import Dict, List

import numpy as np

import plain_zusotar as plain
from plain_qwen2 import read_safetensors


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, top, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def _latent(heads, dim, rot_dim, vdim, kv_rank, base, scale, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim}}}


def _window(heads, kv_heads, dim, vdim, size, scale, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": scale}}


def _gla(heads, dim, vdim, tau, rank, mlp=None):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "a_rank": rank}}


def _config(vocab, width, positions, eps, mult, layers):
    return {"architecture": "Zusotar", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": eps},
            "residual_mult": mult, "layers": layers}


# S1: sizes that vector widths and tensor-core tiles divide; every mixer, dense and routed feed-forwards, two windows.
S1 = _config(300, 64, 320, 1e-5, 0.4, [
    _latent(4, 32, 16, 16, 48, 1000.0, 0.25, mlp=_moe(32, 8, 3, groups=(4, 2), shared=48)),
    _gla(2, 32, 16, 8.0, 16, mlp=_dense(96)),
    _window(4, 2, 32, 16, 24, 0.3, mlp=_moe(32, 6, 2, groups=(2, 1))),
    _gla(4, 16, 32, 3.0, 8, mlp=None),
    _window(2, 1, 16, 32, 9, 0.2, mlp=_moe(16, 4, 4, shared=32)),
])

# S2: sizes that no vector width and no tile divides, a last layer that is a latent attention, groups of one expert, as
# many key heads as heads, a contribution factor of 1.
S2 = _config(101, 100, 290, 1e-6, 1.0, [
    _window(3, 3, 20, 14, 7, 0.4, mlp=_dense(50)),
    _latent(5, 12, 6, 10, 22, 77.0, 0.3, mlp=_moe(30, 5, 2, groups=(5, 3), shared=10)),
    _gla(3, 12, 22, 1.0, 5, mlp=_moe(18, 3, 1)),
    _latent(1, 30, 10, 34, 26, 9.0, 0.2, mlp=None),
])

# S3: one head with more value channels than a tile of the scan's kernels, six query heads over one key head, a window of
# one, all experts of the kept groups chosen, a recurrence last, a factor above 1.
S3 = _config(515, 128, 300, 1e-6, 1.7, [
    _gla(1, 48, 144, 16.0, 24, mlp=_moe(64, 9, 6, groups=(3, 2), shared=32)),
    _window(6, 1, 16, 48, 1, 0.25, mlp=_dense(72)),
    _latent(2, 64, 32, 48, 80, 500000.0, 0.1, mlp=_moe(32, 2, 1, groups=(1, 1))),
    _gla(2, 40, 40, 2.0, 16, mlp=_moe(48, 4, 2, groups=(2, 2))),
])

CASES = {"S1": (S1, 61), "S2": (S2, 62), "S3": (S3, 63)}


def loud(tensors: Dict[str, "torch.Tensor"], seed: int) -> None:
    """Random weights under which every mechanism shows: averages over depth that lean on the last result but take something
    of all, biases by distance from slight to strong, sinks of the scores' size, decays from short to long memories."""
    import torch
    rng = np.random.default_rng(seed)
    for name in sorted(tensors):
        t, leaf = tensors[name], name.split(".", 1)[-1]
        if leaf == "dwa":
            v = rng.normal(0, 0.1, t.numel())
            v[-1] += 0.8
        elif name in ("embed", "pos"):
            v = rng.normal(0, 0.8, t.shape)
        elif leaf == "mix.r1":
            v = rng.uniform(0.05, 2.5, t.numel())
        elif leaf == "mix.r2":
            v = rng.uniform(0.05, 0.5, t.numel())
        elif leaf == "mix.sink":
            v = rng.normal(1.0, 1.5, t.numel())
        elif leaf == "mix.a2.b":
            v = rng.uniform(-1.5, 6.0, t.numel())
        else:
            continue
        tensors[name] = torch.tensor(v, dtype=torch.float32).to(t.dtype)


def make_folder(tmp_path, name: str, config=None, seed=None) -> str:
    import torch
    from coheryn_ai_studio_b200.config.zusotar import ZusotarConfig, zusotar_model_spec
    from coheryn_ai_studio_b200.parts.base import Runtime
    from coheryn_ai_studio_b200.parts.model import DecoderModel
    from coheryn_ai_studio_b200.weights.loader import InitPolicy, random_tensors, write_model_folder
    cfg, s = CASES[name] if config is None else (config, seed)
    c = ZusotarConfig.from_dict(cfg)
    specs = DecoderModel(zusotar_model_spec(c), Runtime(torch.bfloat16, torch.device("cpu"))).tensor_specs()
    tensors = random_tensors(specs, s, InitPolicy(matrix_std=1.0 / c.width ** 0.5, bias_std=0.4, norm_jitter=0.1))
    loud(tensors, s)
    d = str(tmp_path / f"zusotar_{name}")
    write_model_folder(d, c.to_dict(), tensors)
    return d


def read_model(folder: str):
    with open(f"{folder}/config.json") as f:
        config = json.load(f)
    return config, {k: np.asarray(v, dtype=np.float64) for k, v in read_safetensors(f"{folder}/model.safetensors").items()}


_rows: Dict[tuple, np.ndarray] = {}


def plain_rows(folder: str, tokens: List[int], rounded: bool = False) -> np.ndarray:
    key = (folder, tuple(tokens), rounded)
    if key not in _rows:
        config, w = read_model(folder)
        _rows[key] = plain.forward(tokens, w, config, rounded=rounded)
    return _rows[key]


def clear_rows(folder: str, tokens: List[int]) -> np.ndarray:
    """Per position whether no router of the plain model rests on a close call there."""
    key = (folder, tuple(tokens), "clear")
    if key not in _rows:
        config, w = read_model(folder)
        margins = []
        plain.forward(tokens, w, config, margins=margins)
        _rows[key] = np.min(margins, axis=0) > CLEAR if margins else np.ones(len(tokens), dtype=bool)
    return _rows[key]


# float32: only the order of sums differs.  bfloat16: the weights are the same bits, activations are rounded to eight bits
# of mantissa between the kernels; what that costs a row by itself is measured on the plain model's rounded twin, and an
# engine row may be a small factor further from the unrounded row than the twin is (``replay.bf16_excess``).  A router's
# choice between two experts (or groups) whose scores nearly tie can fall the other way after rounding, in the twin and in
# the engine at different rows; such a row is far from the unrounded one, and the rows behind it see it through the mixers.
# So the sequences are made without close calls (``clear_prompt``), what rests on one all the same is left out, and over the
# rows of a test the median is within the bound and at most one in ten (or two) beyond one and a half bounds.
CLEAR = 0.012
TOL_F32 = 2e-4
WORST = {"float32": 0.0, "bfloat16": 0.0}


def check_rows(rows: Dict[tuple, np.ndarray], folder: str, sequences: Dict[str, List[int]], dtype: str, label: str = ""):
    from replay import bf16_excess
    assert rows, "nothing was compared"
    excesses = []
    for (rid, pos), row in sorted(rows.items()):
        ref = plain_rows(folder, sequences[rid])[pos]
        if dtype == "float32":
            d = np.abs(row.astype(np.float64) - ref).max()
            WORST[dtype] = max(WORST[dtype], float(d) / max(1.0, float(np.std(ref))))
            assert d <= TOL_F32 * max(1.0, float(np.std(ref))), f"{label} {rid}@{pos}: |d| = {d:.3e}"
        elif clear_rows(folder, sequences[rid])[pos]:
            twin = plain_rows(folder, sequences[rid], rounded=True)[pos]
            excesses.append((bf16_excess(row, ref.astype(np.float32), twin.astype(np.float32)), rid, pos))
    if dtype != "float32" and len(rows) > 4:
        assert 2 * len(excesses) >= len(rows), f"{label}: only {len(excesses)} of {len(rows)} rows are clear of close calls"
    if excesses:
        values = np.array([e[0] for e in excesses])
        WORST[dtype] = max(WORST[dtype], float(np.median(values)))
        far = int((values > 1.5).sum())
        assert np.median(values) <= 1.0, f"{label}: median {np.median(values):.2f} of the bfloat16 bound"
        assert far <= max(2, len(values) // 10), f"{label}: {far} of {len(values)} rows beyond 1.5 bounds (worst {max(excesses)})"


def noisy_replay(folder: str, dtype: str, max_tokens: int, model, max_requests: int = 4, page_size: int = 16, **kw):
    """The replay harness with the state slots full of noise as well as the pages."""
    from replay import Replay
    r = Replay(folder, dtype, max_tokens=max_tokens, model=model, max_requests=max_requests, page_size=page_size, **kw)
    for t in r.cache.state_tensors():
        t.normal_(0.0, 4.0)
    return r


def prompt(seed: int, n: int, vocab: int) -> List[int]:
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


_prompts: Dict[tuple, List[int]] = {}


def clear_prompt(folder: str, seed: int, n: int) -> List[int]:
    """``n`` random tokens of which hardly one makes a router of the plain model choose by a hair: those that do are drawn
    again, a few times over."""
    key = (folder, seed, n)
    if key not in _prompts:
        vocab = read_model(folder)[0]["vocab"]
        rng = np.random.default_rng(seed)
        tokens = rng.integers(0, vocab, size=n)
        for _ in range(8):
            close = ~clear_rows(folder, tokens.tolist())
            if not close.any():
                break
            tokens[close] = rng.integers(0, vocab, size=int(close.sum()))
        _prompts[key] = tokens.tolist()
    return _prompts[key]
