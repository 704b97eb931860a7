"""Small configurations of the Gebasun decoder for tests.  They differ from one another in every size and option: head
counts and key/value groups (one to as many as heads), head sizes the tiled attention kernels take and others, windows
shorter than a page, at a page's edge and longer, kept first tokens within a page and beyond one, no mask at all, distance
tables whose scale ends inside and beyond the window, rotations over two dimensions and whole heads, state-space layers
with one group, one group per head and in between, one to five taps, odd head and state sizes, norms in one part and in
several, one chosen expert to all of them, layers without a feed-forward and without a shared expert, widths that are no
multiple of eight."""


def _moe(ff, experts, top, shared):
    m = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if shared:
        m["shared"] = dict(ff=shared)
    return m


def _biased(heads, kv_heads, dim, scale, window, bias_max, rows, mlp):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale, bias_max=bias_max, bias_rows=rows)
    if window:
        m["mask"] = dict(size=window)
    return dict(type="attention", mixer=m, mlp=mlp)


def _rotated(heads, kv_heads, dim, scale, window, keep, dims, base, mlp):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale, rot=dict(dims=dims, base=base))
    if window:
        m["mask"] = dict(size=window, keep_first=keep)
    return dict(type="attention_2", mixer=m, mlp=mlp)


def _ssm(heads, vdim, state, groups, conv, norm_groups, mlp):
    return dict(type="mamba2", mlp=mlp, mixer=dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv,
                                                   norm_groups=norm_groups))


# General head sizes, windows within a page, kept tokens beyond one, a layer without a feed-forward, a distance scale that
# ends inside the window.
GB_A = dict(
    architecture="Gebasun", vocab=211, width=96, norm=dict(eps=1e-5),
    layers=[
        _rotated(4, 2, 24, 0.25, 37, 70, 8, 1000.0, _moe(40, 6, 2, 24)),
        _ssm(4, 20, 12, 2, 3, 4, _moe(24, 5, 1, 48)),
        _biased(6, 3, 20, 0.3, 50, 33, 10, _moe(32, 4, 4, 16)),
        _ssm(3, 24, 18, 1, 5, 1, None),
    ])
# A width that is no multiple of eight (every product on the FMA units), odd head, state and expert sizes, one tap, a group
# per head, no mask, no shared expert, eps that shows.
GB_B = dict(
    architecture="Gebasun", vocab=300, width=100, norm=dict(eps=1e-3),
    layers=[
        _ssm(5, 13, 7, 5, 1, 5, _moe(20, 7, 3, 0)),
        _biased(3, 1, 18, 0.2, None, 90, 7, _moe(36, 3, 2, 20)),
        _rotated(6, 6, 14, 0.4, None, 0, 14, 100.0, _moe(12, 9, 5, 28)),
        _ssm(2, 9, 30, 1, 2, 3, _moe(28, 2, 1, 12)),
    ])
# The sizes the tiled kernels like: heads of 64 and 128, windows at and across pages, states of 64 and 128, experts on the
# tensor cores.
GB_C = dict(
    architecture="Gebasun", vocab=512, width=256, norm=dict(eps=1e-6),
    layers=[
        _ssm(8, 64, 64, 2, 4, 2, _moe(64, 8, 2, 128)),
        _biased(4, 1, 128, 0.1, 100, 300, 32, _moe(128, 4, 2, 64)),
        _rotated(8, 4, 64, 0.2, 64, 3, 32, 10000.0, _moe(64, 16, 4, 64)),
        _biased(8, 8, 64, 0.15, 129, 64, 16, None),
        _rotated(4, 2, 128, 0.09, 150, 65, 128, 500000.0, _moe(72, 6, 3, 136)),
        _ssm(2, 128, 128, 1, 4, 1, _moe(64, 8, 8, 64)),
    ])
# Decode kernels at sizes between, more query heads than one group of eight, many state-space heads of few columns, a norm
# whose parts cut through heads, a table of two rows.
GB_D = dict(
    architecture="Gebasun", vocab=1000, width=184, norm=dict(eps=1e-4),
    layers=[
        _biased(18, 2, 32, 0.2, 200, 150, 2, _moe(48, 12, 3, 56)),
        _ssm(12, 8, 96, 4, 4, 3, _moe(40, 5, 2, 72)),
        _rotated(10, 5, 80, 0.15, 90, 1, 2, 30.0, _moe(64, 8, 1, 40)),
        _ssm(6, 36, 68, 3, 3, 8, None),
        _biased(4, 4, 112, 0.12, 65, 2000, 40, _moe(24, 10, 6, 16)),
    ])
ALL = {"A": GB_A, "B": GB_B, "C": GB_C, "D": GB_D}


def make_folder(tmp_path, name: str, dtype: str, seed: int = 4321):
    from pathlib import Path

    from llmoxide_b200.config import read_config
    from llmoxide_b200.weights import write_model_folder

    cfg = dict(ALL[name], torch_dtype=dtype)
    folder = Path(tmp_path) / f"gebasun_{name}_{dtype}"
    if not (folder / "model.safetensors").exists():
        write_model_folder(folder, read_config(cfg), seed, dtype)
    return folder
