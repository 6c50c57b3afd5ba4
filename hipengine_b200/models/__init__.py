"""models subpackage."""


def make_executor(weights, dtype: str = "bfloat16", **kw):
    """Executor of the checkpoint's family.  ``dtype``: compute precision (``float32`` where the family declares it)."""
    from .registry import load_object, plugin_for
    plugin = plugin_for(weights.config.arch)
    if dtype not in plugin.compute_dtypes:
        raise ValueError(f"{plugin.name}: compute dtype {dtype!r} is not built (supported: {plugin.compute_dtypes})")
    if len(plugin.compute_dtypes) > 1:
        kw["dtype"] = dtype
    return load_object(plugin.executor)(weights, **kw)
