"""Small configurations of the Soputar decoder for tests.  They differ from one another in every size and option:
head counts and key/value groups (one to as many as heads), key and value sizes that differ and that agree, a query
temperature that steps every position and one that never steps, capped scores that bind and none, borrowed keys and
values (twice from one layer, with constants of their own), latents wider and narrower than the heads, one to five
convolution taps, delta heads that share a key head and that do not, layers without a feed-forward, widths that are no
multiple of eight, and sizes that the tiled attention kernels take."""


def _attention(heads, kv_heads, dim, vdim, scale, softcap, temp, ff, limit=3.0, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if softcap is not None:
        m["softcap"] = softcap
    if temp is not None:
        m["q_temp"] = dict(coef=temp[0], every=temp[1])
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m, mlp=_mlp(ff, limit))


def _latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, ff, limit=3.0):
    return dict(type="latent_attention", mlp=_mlp(ff, limit),
                mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale,
                           rot=dict(base=base, dims=rot_dim)))


def _delta(heads, kv_heads, dim, vdim, conv, ff, limit=3.0):
    return dict(type="delta", mlp=_mlp(ff, limit), mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv))


def _mlp(ff, limit):
    return None if ff is None else dict(kind="dense", ff=ff, limit=limit)


# The delta rule first; values narrower than keys; two key/value groups; a cap that binds; a temperature that steps every
# three positions; a borrower with a scale, a cap and a temperature of its own; a layer without a feed-forward.
SP_A = dict(
    architecture="Soputar", vocab=211, width=96, norm=dict(eps=1e-5), embedding=dict(scale=3.0),
    layers=[
        _delta(4, 2, 24, 16, 3, 40, limit=1.5),
        _attention(4, 2, 32, 16, 0.3, 2.5, (0.4, 3), 72, limit=0.7),
        _latent(3, 16, 8, 24, 40, 0.25, 1000.0, 56),
        _attention(6, 2, 32, 16, 0.5, 6.0, (0.2, 20), None, kv_from=1),
    ])
# A width that is no multiple of eight (every product on the FMA units), one tap (no convolution beyond the current
# token), values wider than keys, no cap, no temperature, six delta heads on three key heads, an odd head size.
SP_B = dict(
    architecture="Soputar", vocab=300, width=100, norm=dict(eps=1e-6), embedding=dict(scale=0.5),
    layers=[
        _latent(5, 20, 12, 12, 28, 0.3, 50000.0, 36),
        _attention(6, 3, 16, 48, 0.25, None, None, 44, limit=10.0),
        _delta(6, 3, 30, 41, 1, None),
        _attention(3, 3, 48, 40, 0.15, 1.0, (0.9, 1), 30),
    ])
# The sizes the tiled kernels like (64 and 128): capped and plain scores, one kv head, borrowed keys, assembled latent
# keys of 128 and of 64 with values of the same size, delta heads of 128 and 64 sharing key heads.
SP_C = dict(
    architecture="Soputar", vocab=512, width=256, norm=dict(eps=1e-6), embedding=dict(scale=1.0),
    layers=[
        _attention(4, 1, 128, 128, 0.2, 4.0, (0.3, 40), 128),
        _latent(4, 96, 32, 128, 144, 0.12, 10000.0, 256),
        _delta(4, 2, 128, 128, 4, 128),
        _attention(8, 4, 64, 64, 0.3, 3.0, (0.5, 16), 128),
        _attention(4, 1, 128, 128, 0.15, None, None, 160, kv_from=0),
        _delta(6, 2, 64, 64, 2, None),
        _latent(2, 48, 16, 64, 80, 0.2, 500.0, 128),
        _attention(8, 4, 64, 64, 0.125, None, (0.1, 7), 96, kv_from=3),
    ])
# Sizes that are no power of two, a latent far wider than its heads, more heads than one tile of sixteen, five taps,
# as many key/value heads as heads, delta keys beyond 128.
SP_D = dict(
    architecture="Soputar", vocab=1000, width=184, norm=dict(eps=1e-4), embedding=dict(scale=7.5),
    layers=[
        _latent(20, 8, 16, 24, 304, 0.22, 100.0, 72),
        _attention(6, 2, 96, 32, 0.2, 5.0, (0.7, 64), 100),
        _delta(3, 3, 140, 20, 5, 72),
        _attention(8, 8, 24, 24, 0.3, 1.5, (0.25, 50), 33),
        _attention(16, 8, 24, 24, 0.2, None, None, 72, kv_from=3),
        _delta(8, 1, 32, 72, 4, 40),
    ])
ALL = {"A": SP_A, "B": SP_B, "C": SP_C, "D": SP_D}


def make_folder(tmp_path, name: str, dtype: str, seed: int = 4321):
    from pathlib import Path

    from llmoxide_b200.config import read_config
    from llmoxide_b200.weights import write_model_folder

    cfg = dict(ALL[name], torch_dtype=dtype)
    folder = Path(tmp_path) / f"soputar_{name}_{dtype}"
    if not (folder / "model.safetensors").exists():
        write_model_folder(folder, read_config(cfg), seed, dtype)
    return folder
