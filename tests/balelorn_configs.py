"""Tiny Balelorn configurations that differ from each other in every size, constant and in the order of layers, and
the helper that writes a folder of random weights for one (into a temporary folder, never committed)."""
from __future__ import annotations

ARCH = "Balelorn"


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def attention(heads, kv_heads, dim, vdim, scale, mlp, chunk=None, rot=None, v_mix=False):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


# A: sizes in steps of 16; chunks of 24 (no multiple of the pages' 8 positions in every layer: 24, 21, 50); the first
# layer does not mix its values, the second is the source; experts first, a dense layer behind them.
BALELORN_A = {
    "architecture": ARCH, "vocab": 211, "width": 64, "norm": {"eps": 1e-5},
    "layers": [
        attention(4, 2, 32, 48, 0.2, moe(6, 2, 32, 1.5), chunk=24, rot=(16, 500.0)),
        attention(2, 1, 48, 32, 0.15, dense(96), chunk=21, rot=(48, 10000.0), v_mix=True),
        attention(4, 2, 16, 16, 0.3, moe(5, 1, 48, 7.0), chunk=24, rot=(8, 77.0), v_mix=True),
        attention(8, 1, 32, 32, 0.25, None, chunk=50, rot=(32, 20000.0), v_mix=True),
    ],
}

# B: sizes that are no multiple of 16 or 8 (the warp-per-row attention in both engines), as many key heads as query
# heads, a chunk of one position, a layer without chunks and one without rotation, all experts chosen, no feed-forward
# in the middle, values mixed from the first layer on.
BALELORN_B = {
    "architecture": ARCH, "vocab": 97, "width": 72, "norm": {"eps": 3e-6},
    "layers": [
        attention(3, 3, 20, 12, 0.35, dense(50), chunk=13, rot=(6, 1000.0), v_mix=True),
        attention(6, 1, 12, 36, 0.15, None, rot=(12, 33.0), v_mix=True),
        attention(2, 2, 24, 20, 0.4, moe(3, 3, 24, 0.8), chunk=1),
        attention(9, 3, 10, 12, 0.3, moe(7, 2, 40, 2.5), chunk=37, rot=(4, 250000.0), v_mix=True),
    ],
}

# C: larger heads at the page size of serving, where the kernels that stream pages by TMA run: keys and values of 64,
# of 128, and of different widths; chunks at, beside and across the pages' 64 positions.
BALELORN_C = {
    "architecture": ARCH, "vocab": 131, "width": 128, "norm": {"eps": 1e-6},
    "layers": [
        attention(8, 2, 64, 64, 0.11, moe(8, 3, 96, 2.0), chunk=64, rot=(32, 20000.0), v_mix=True),
        attention(4, 1, 128, 128, 0.07, dense(160), chunk=100, rot=(128, 250000.0), v_mix=True),
        attention(6, 3, 96, 40, 0.09, moe(8, 3, 64, 3.0), chunk=129, rot=(48, 500.0)),
        attention(4, 2, 128, 64, 0.08, moe(4, 2, 96, 1.0), chunk=90, rot=(64, 10000.0), v_mix=True),
    ],
}

CONFIGS = {"A": (BALELORN_A, 51), "B": (BALELORN_B, 52), "C": (BALELORN_C, 53)}
STD = {"A": 0.2, "B": 0.2, "C": 0.12}


def make_folder(tmp_path, name, std=None):
    from ferrox_b200 import write_random_model

    cfg, seed = CONFIGS[name]
    folder = str(tmp_path / f"balelorn_{name}")
    write_random_model(folder, cfg, seed, dtype="bfloat16", std=std or STD[name], norm_init="around_one")
    return folder
