"""Tiny Bogivik configurations for the tests.  They differ in every size and option: both kinds of layer in several orders,
query heads that share key/value heads and that do not, value heads smaller, larger than and equal to the query/key heads,
turned spans from 2 entries to a whole head and none, stretched and plain frequencies, chunks from one key to more than the
prompts hold and none, bucket counts from 2 to 32 with farthest distances from a few keys to more than the prompts hold, layers
with and without a query temperature, with and without mixed values (the first such layer not always the first layer),
memory heads on every width of the recurrence kernel, gate caps from 1 to 20, layers without a feed-forward, and models of one
kind of layer alone."""
import os


def _attention(heads, kv, dim, vdim, scale, rows, farthest, temp=None, v_mix=False):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "bias_rows": rows, "bias_max": farthest, "v_mix": v_mix}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m}


def _left(heads, kv, dim, vdim, scale, chunk, dims, base, scaling=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk} if chunk else None,
         "rot": {"base": base, "dims": dims}}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def _parallel(left, heads, dim, vdim, cap):
    return {"type": "parallel", "mixer": {"left": left, "right": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}}


def _with(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff} if ff else None)


# grouped heads on both kinds of layer, values smaller and larger than keys, the first v_mix layer behind a parallel one
BG_A = {
    "architecture": "Bogivik", "vocab": 211, "width": 96, "norm": {"eps": 1e-5},
    "layers": [
        _with(_parallel(_left(4, 2, 32, 16, 0.2, 13, 16, 5000.0, (4.0, 1.0, 4.0, 64)), 3, 16, 24, 6.0), 80),
        _with(_attention(4, 2, 16, 24, 0.3, 16, 40, (0.4, 16), v_mix=True), 48),
        _with(_parallel(_left(2, 2, 16, 40, 0.3, 29, 8, 300.0), 2, 24, 8, 12.0), None),
        _with(_attention(6, 3, 24, 16, 0.25, 8, 100.5, None, v_mix=True), 64),
        _with(_attention(2, 1, 32, 32, 0.2, 6, 9, (0.2, 3)), None),
    ],
}
# the tensor-core attention kernels: rows of 64 and 128 with pages of 16
BG_B = {
    "architecture": "Bogivik", "vocab": 500, "width": 128, "norm": {"eps": 1e-6},
    "layers": [
        _with(_attention(2, 1, 64, 64, 0.125, 32, 70, (0.3, 32), v_mix=True), 160),
        _with(_parallel(_left(4, 4, 128, 128, 0.09, 40, 64, 20000.0, (8.0, 1.0, 4.0, 128)), 2, 32, 64, 10.0), None),
        _with(_attention(8, 1, 64, 64, 0.14, 10, 400, None, v_mix=True), 96),
        _with(_parallel(_left(4, 2, 64, 128, 0.11, 33, 24, 2e5, (2.0, 2.0, 3.0, 30)), 3, 40, 64, 20.0), 64),
        _with(_attention(2, 2, 128, 128, 0.088, 4, 21, (0.5, 8)), 64),
    ],
}
# sizes that fit no vector width, a width that is a multiple of 4 only, chunks of 3, two buckets
BG_C = {
    "architecture": "Bogivik", "vocab": 173, "width": 52, "norm": {"eps": 1e-4},
    "layers": [
        _with(_attention(3, 3, 20, 12, 0.3, 2, 5, (0.3, 1), v_mix=True), 36),
        _with(_parallel(_left(3, 3, 18, 26, 0.3, 3, 2, 77.0, (3.0, 1.0, 8.0, 20)), 1, 40, 20, 3.0), 40),
        _with(_attention(6, 3, 10, 12, 0.4, 12, 30, None, v_mix=True), None),
        _with(_parallel(_left(6, 2, 14, 8, 0.25, 500, 12, 900.0), 5, 8, 12, 8.0), 20),
    ],
}
# attention layers alone (no state slot at all), no mixed values
BG_D = {
    "architecture": "Bogivik", "vocab": 150, "width": 64, "norm": {"eps": 1e-5},
    "layers": [
        _with(_attention(2, 1, 40, 40, 0.2, 14, 33, (1.5, 5)), 48),
        _with(_attention(4, 4, 8, 72, 0.5, 32, 1000, None), None),
        _with(_attention(12, 2, 16, 16, 0.3, 20, 60, (0.2, 700)), 32),
    ],
}
# parallel layers alone; memory keys of 136 and 256 entries; no mask
BG_E = {
    "architecture": "Bogivik", "vocab": 99, "width": 72, "norm": {"eps": 1e-6},
    "layers": [
        _with(_parallel(_left(2, 1, 16, 24, 0.3, 17, 8, 100.0, (4.0, 1.0, 4.0, 40)), 1, 136, 4, 5.0), 36),
        _with(_parallel(_left(1, 1, 8, 8, 0.4, None, 4, 10.0), 2, 256, 4, 1.0), None),
        _with(_parallel(_left(3, 1, 24, 24, 0.2, 64, 24, 1000.0, (16.0, 1.0, 2.0, 16)), 8, 12, 36, 15.0), 24),
    ],
}
# ones and extremes: single heads, chunks of one key (a token sees itself alone) and of two, a feed-forward of 8, a memory of 4 x 4
BG_F = {
    "architecture": "Bogivik", "vocab": 64, "width": 48, "norm": {"eps": 1e-6},
    "layers": [
        _with(_parallel(_left(1, 1, 8, 8, 1.0, 1, 8, 10.0), 1, 4, 4, 4.0), 8),
        _with(_attention(1, 1, 8, 8, 1.0, 2, 2, (1.0, 1), v_mix=True), None),
        _with(_parallel(_left(1, 1, 8, 8, 0.7, 2, 8, 10.0, (2.0, 1.0, 4.0, 8)), 1, 8, 8, 2.0), 8),
        _with(_attention(1, 1, 8, 8, 0.6, 4, 7, None, v_mix=True), 8),
    ],
}
CONFIGS = {"A": (BG_A, 61), "B": (BG_B, 62), "C": (BG_C, 63), "D": (BG_D, 64), "E": (BG_E, 65), "F": (BG_F, 66)}
INIT_SCALE = 5.0


def make_model_dir(tmp_root, name, dtype="bfloat16"):
    """Write the folder with the framework's random-weights writer."""
    from zedinfer_b200.weights import write_random_model
    cfg, seed = CONFIGS[name]
    out = os.path.join(str(tmp_root), f"bogivik_{name}_{dtype}")
    if not os.path.isfile(os.path.join(out, "model.safetensors")):
        write_random_model(cfg, seed, out, dtype=dtype, init_scale=INIT_SCALE, name_prefix="")
    return out
