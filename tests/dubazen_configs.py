"""Tiny Dubazen configurations that differ from each other in every size, constant and in the order of layers, and the
helper that writes a folder of random weights for one (into a temporary folder, never committed)."""
from __future__ import annotations

ARCH = "Dubazen"


def moe(experts, top, ff, limit, shared_ff=None, shared_limit=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared_ff:
        m["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return m


def attention(heads, kv_heads, dim, vdim, scale, rot):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
            "rot": {"dims": rot[0], "base": rot[1]}}


def lightning(dim, vdim, decay):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}


def parallel(left, right, scales, mlp):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "right": right, "left_scale": scales[0],
                                                      "right_scale": scales[1]}}


def gla(heads, dim, vdim, tau, mlp):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def mamba(inner, state, dt_rank, conv, mlp):
    return {"type": "mamba1", "mlp": mlp, "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}


# A: sizes in steps of 16, two streams; a parallel layer first and last.
DUBAZEN_A = {
    "architecture": ARCH, "vocab": 211, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0}, "streams": 2,
    "layers": [
        parallel(attention(4, 2, 32, 48, 0.3, (16, 500.0)), lightning(16, 32, (0.7, 0.97)), (0.8, 1.1), moe(6, 2, 32, 1.5, 48, 0.9)),
        mamba(96, 16, 8, 4, moe(5, 1, 48, 2.5, 32, 7.0)),
        gla(4, 16, 32, 16.0, None),
        parallel(attention(2, 1, 48, 16, 0.4, (48, 10000.0)), lightning(32, 16, (0.5, 0.9, 0.999)), (1.0, 0.3), moe(4, 4, 16, 1.0)),
    ],
}

# B: sizes that are no multiple of 16 or 8 (the warp-per-row attention in both engines), five streams, as many key heads
# as query heads, one head, one state a channel, other numbers of taps, no rotation of queries and keys in one layer, all
# experts chosen, no shared expert, layers without a feed-forward first and in the middle.
DUBAZEN_B = {
    "architecture": ARCH, "vocab": 97, "width": 72, "norm": {"eps": 3e-6}, "embedding": {"scale": 1.0}, "streams": 5,
    "layers": [
        gla(1, 20, 12, 1.0, None),
        parallel(attention(3, 3, 20, 10, 0.35, (6, 1000.0)), lightning(12, 20, (0.9,)), (1.3, 1.0), moe(3, 3, 24, 0.8)),
        mamba(50, 1, 3, 2, moe(7, 2, 40, 1.5, 20, 2.0)),
        parallel(attention(6, 1, 12, 36, 0.5, (0, 33.0)), lightning(20, 6, (0.4, 0.95, 0.6, 0.8)), (0.5, 2.0), None),
        mamba(36, 6, 5, 3, None),
        gla(3, 36, 24, 4.0, moe(5, 2, 20, 1.2, 28, 1.1)),
    ],
}

# C: larger heads at the page size of serving, where the kernels that stream pages by TMA run: keys and values of 128,
# of 64, and of different widths; three streams; a state of 128 x 64 a head.
DUBAZEN_C = {
    "architecture": ARCH, "vocab": 131, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 11.3}, "streams": 3,
    "layers": [
        mamba(256, 16, 16, 4, moe(8, 3, 96, 2.0, 160, 3.0)),
        parallel(attention(4, 1, 128, 128, 0.2, (64, 20000.0)), lightning(64, 128, (0.9, 0.99)), (1.0, 1.0), moe(8, 2, 64, 3.0, 64, 1.0)),
        gla(2, 128, 64, 16.0, moe(8, 3, 96, 2.0, 96, 2.0)),
        parallel(attention(8, 2, 64, 64, 0.25, (64, 250000.0)), lightning(128, 64, (0.95, 0.8)), (0.6, 1.4), moe(4, 2, 96, 1.0, 32, 1.0)),
        parallel(attention(4, 2, 128, 96, 0.15, (32, 10000.0)), lightning(32, 32, (0.9, 0.9, 0.99)), (1.0, 0.5), None),
    ],
}

CONFIGS = {"A": (DUBAZEN_A, 61), "B": (DUBAZEN_B, 62), "C": (DUBAZEN_C, 63)}
STD = {"A": 0.15, "B": 0.15, "C": 0.08}


def make_folder(tmp_path, name, std=None):
    from ferrox_b200 import write_random_model

    cfg, seed = CONFIGS[name]
    folder = str(tmp_path / f"dubazen_{name}")
    write_random_model(folder, cfg, seed, dtype="bfloat16", std=std or STD[name], norm_init="around_one")
    return folder
