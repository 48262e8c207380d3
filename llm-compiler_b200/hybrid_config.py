"""What the configurations of the hybrid designs share."""


class ConfigError(ValueError):
    """config.json asks for something the design does not have, or contradicts itself."""
