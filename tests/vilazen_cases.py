"""Small Vilazen configurations of the tests (they differ from each other in every size and option), folders of seeded
random weights for them, and the comparison of engine rows with the plain implementation."""
from __future__ import annotations

import json
from typing import Dict, List

import numpy as np

import plain_vilazen as plain
from plain_qwen2 import read_safetensors


def _mlp(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def _window(heads, kv_heads, dim, vdim, size, keep, dims, base, scale, ff, mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}, "v_mix": mix}
    if size is not None:
        m["mask"] = {"size": size} if keep is None else {"size": size, "keep_first": keep}
    return {"type": "attention", "mixer": m, "mlp": _mlp(ff)}


def _latent(heads, dim, rot_dim, vdim, kv_rank, size, base, scale, ff):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    if size is not None:
        m["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": m, "mlp": _mlp(ff)}


def _both(left, right, scales, ff):
    """left: (heads, kv_heads, dim, vdim, rotated channels, base, scale); right: (dim, vdim, decays)."""
    H, G, dk, dv, dims, base, scale = left
    return {"type": "parallel", "mlp": _mlp(ff), "mixer": {
        "left": {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": scale, "rot": {"base": base, "dims": dims}}, "left_scale": scales[0],
        "right": {"heads": len(right[2]), "dim": right[0], "vdim": right[1], "decay": list(right[2])}, "right_scale": scales[1]}}


def _config(vocab, width, eps, layers):
    return {"architecture": "Vilazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# V1: sizes that vector widths and tensor-core tiles divide; every mixer; a layer that mixes no values between those that do;
# the first of them is not the model's first layer.
V1 = _config(300, 64, 1e-5, [
    _both((4, 2, 32, 16, 16, 1000.0, 0.25), (16, 32, [0.5, 0.97, 1.0]), (0.7, 0.4), 96),
    _window(4, 2, 32, 16, 24, 5, 32, 500.0, 0.3, 64),
    _window(2, 1, 16, 48, 11, 16, 8, 90.0, 0.35, None, mix=False),
    _latent(4, 32, 16, 16, 48, 21, 1000.0, 0.25, 128),
    _window(8, 1, 16, 32, 40, 0, 16, 10000.0, 0.3, 80),
])

# V2: sizes that no vector width and no tile divides (the output products of a layer cannot be joined), a window of one with
# one kept position, an attention without a mask, a latent attention last, negative and large factors.
V2 = _config(101, 100, 1e-6, [
    _window(3, 3, 20, 14, 7, 3, 6, 77.0, 0.4, 50),
    _both((6, 2, 10, 22, 10, 30.0, 0.5), (12, 7, [0.0, 0.9]), (-1.3, 2.0), 30),
    _window(6, 3, 12, 14, 1, 1, 12, 9.0, 0.5, 22),
    _window(2, 1, 18, 10, None, None, 4, 300.0, 0.3, None, mix=False),
    _latent(5, 12, 6, 10, 22, 9, 77.0, 0.3, 18),
])

# V3: windows shorter than what they keep, more query heads than a decode tile over one key head, one linear-attention head
# with more value channels than a tile, two mixers side by side last.
V3 = _config(515, 128, 1e-6, [
    _window(18, 1, 16, 16, 6, 37, 16, 50.0, 0.25, 192),
    _latent(2, 64, 32, 48, 80, None, 500000.0, 0.1, 64),
    _window(2, 2, 64, 8, 64, 64, 48, 1e6, 0.125, 40),
    _both((2, 2, 64, 48, 64, 20000.0, 0.125), (48, 144, [0.999]), (0.5, 0.6), 72),
])

CASES = {"V1": (V1, 81), "V2": (V2, 82), "V3": (V3, 83)}


def loud(tensors: Dict[str, "torch.Tensor"], seed: int) -> None:
    """Random weights under which every mechanism shows: sinks of the scores' size, shares of the first layer's values far
    from 0 and 1, biases that matter."""
    import torch
    rng = np.random.default_rng(seed)
    for name in sorted(tensors):
        t, leaf = tensors[name], name.split(".", 1)[-1]
        if name == "embed":
            v = rng.normal(0, 1.0, t.shape)
        elif leaf == "mix.left.sink":
            v = rng.normal(1.0, 1.5, t.numel())
        elif leaf == "mix.vmix":
            v = rng.uniform(0.3, 0.7)
        elif leaf in ("mix.left.g", "mix.g", "mix.right.g"):
            v = rng.normal(0, 2.0 / t.shape[1] ** 0.5, t.shape)
        else:
            continue
        tensors[name] = torch.tensor(v, dtype=torch.float32).to(t.dtype)


def make_folder(tmp_path, name: str, config=None, seed=None) -> str:
    import torch
    from coheryn_ai_studio_b200.config.vilazen import VilazenConfig, vilazen_model_spec
    from coheryn_ai_studio_b200.parts.base import Runtime
    from coheryn_ai_studio_b200.parts.model import DecoderModel
    from coheryn_ai_studio_b200.weights.loader import InitPolicy, random_tensors, write_model_folder
    cfg, s = CASES[name] if config is None else (config, seed)
    c = VilazenConfig.from_dict(cfg)
    specs = DecoderModel(vilazen_model_spec(c), Runtime(torch.bfloat16, torch.device("cpu"))).tensor_specs()
    tensors = random_tensors(specs, s, InitPolicy(matrix_std=1.2 / c.width ** 0.5, bias_std=0.4, norm_jitter=0.1))
    loud(tensors, s)
    d = str(tmp_path / f"vilazen_{name}")
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


# float32: only the order of sums differs.  bfloat16: the weights are the same bits, activations are rounded to eight bits
# of mantissa between the kernels; what that costs a row by itself is measured on the plain model's rounded twin, and an
# engine row may be a small factor further from the unrounded row than the twin is (``replay.bf16_excess``).  Over the rows
# of a test at most one in ten (or one) may lie beyond the bound and none beyond one and a half bounds.
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
        else:
            twin = plain_rows(folder, sequences[rid], rounded=True)[pos]
            excesses.append((bf16_excess(row, ref.astype(np.float32), twin.astype(np.float32)), rid, pos))
    if excesses:
        values = np.array([e[0] for e in excesses])
        WORST[dtype] = max(WORST[dtype], float(values.max()))
        over = int((values > 1.0).sum())
        assert values.max() <= 1.5, f"{label}: {max(excesses)} of the bfloat16 bound"
        assert over <= max(1, len(values) // 10), f"{label}: {over} of {len(values)} rows beyond the bfloat16 bound (worst {max(excesses)})"


def noisy_replay(folder: str, dtype: str, max_tokens: int, model, max_requests: int = 4, page_size: int = 16, **kw):
    """The replay harness with the state slots full of noise as well as the pages."""
    from replay import Replay
    r = Replay(folder, dtype, max_tokens=max_tokens, model=model, max_requests=max_requests, page_size=page_size, **kw)
    for t in r.cache.state_tensors():
        t.normal_(0.0, 4.0)
    return r


def prompt(seed: int, n: int, vocab: int) -> List[int]:
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()
