"""Small graphs on the GPU: build a session, feed it, read its outputs, compare."""
import numpy as np


def rng_of(*key):
    return np.random.default_rng(list(key))


def session(g, outputs, params, inputs=None, u32=None):
    import meganeura_b200 as mg
    g.set_outputs(outputs)
    s = mg.build_inference_session(g)
    for n, a in params.items():
        s.set_parameter(n, a)
    for n, a in (inputs or {}).items():
        s.set_input(n, a)
    for n, a in (u32 or {}).items():
        s.set_input_u32(n, a)
    return s


def run(s, *shapes):
    s.step()
    s.wait()
    out = [s.read_output_by_index(i, int(np.prod(sh))).reshape(sh) for i, sh in enumerate(shapes)]
    return out[0] if len(out) == 1 else out


def close(got, want, tol=2e-5):
    want = np.asarray(want)
    assert np.isfinite(got).all()
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)
    assert err <= tol, f"error {err:.3e} > {tol:g}"
